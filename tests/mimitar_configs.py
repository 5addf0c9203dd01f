"""Small Mimitar configurations for the tests: sizes differ from layer to layer and between a layer's two latents, and
values that could hide a fault by being equal (head counts, key and value sizes, the two ranks, the limits of an expert and
of the shared expert) or by being 1 (streams, groups, experts, chosen experts) are mixed on purpose."""

from __future__ import annotations

from layover_b200.config.mimitar import capped_layer, dense_mlp, latent_layer, routed_mlp


def like(layer: dict, index: int) -> dict:
    """A layer that runs with layer `index`'s tensors."""
    return dict(layer, weights_of=index)


def config(vocab, width, streams, layers, mult=1.0, logit_scale=None, eps=1e-5):
    raw = {"architecture": "Mimitar", "vocab": vocab, "width": width, "streams": streams, "residual_mult": mult, "norm": {"eps": eps},
           "layers": layers}
    if logit_scale is not None:
        raw["logit_scale"] = logit_scale
    return raw


def _odd_sizes():
    latent = latent_layer(5, 10, 6, 14, 22, 18, 3000.0, ramp=(5.0, 40, 9.0, 0.7), scale=0.4, mlp=routed_mlp(8, 3, 20, 1.1, (4, 2), (36, 0.8)))
    capped = capped_layer(6, 3, 12, 20, 9000.0, 6, bands=(2.5, 1.0, 3.0, 60), softcap=4.0, scale=0.6, mlp=dense_mlp(44, 0.9))
    return config(211, 74, 3, [latent, capped, like(latent, 0), capped_layer(4, 1, 14, 10, 500.0, 14, softcap=9.0, scale=0.7)], mult=0.7,
                  logit_scale=0.6)


def _wide_heads():
    first = capped_layer(4, 2, 32, 64, 20000.0, 16, bands=(6.0, 1.0, 4.0, 120), softcap=8.0, scale=0.4, mlp=routed_mlp(12, 4, 64, 2.0, (3, 2), (128, 1.5)))
    return config(160, 128, 2, [
        first,
        latent_layer(3, 32, 16, 48, 64, 40, 40000.0, ramp=(3.0, 64, 16.0, 1.0), scale=0.3, mlp=dense_mlp(192, 1.5)),
        capped_layer(2, 1, 128, 128, 10000.0, 128, bands=(9.0, 2.0, 5.0, 200), softcap=5.0, scale=0.1, mlp=dense_mlp(128, 1.2)),
        like(first, 0), like(first, 3),
        # a row of more than 256 channels in the cache; as many heads as two tiles of the decode kernel hold
        latent_layer(17, 16, 8, 8, 272, 24, 700.0, scale=0.5, mlp=routed_mlp(6, 5, 48, 1.0)),
        latent_layer(20, 24, 32, 16, 96, 72, 700.0, ramp=(1.5, 500, 4.0, 1.5), scale=0.35),
    ], mult=0.5, logit_scale=1.7)


def _smallest():
    """One stream, one head, one expert, ranks of 2 and 4; twenty query heads on one key head; a layer that borrows the
    tensors of one behind it."""
    tail = capped_layer(20, 1, 8, 16, 100.0, 2, softcap=6.0, scale=0.5, mlp=routed_mlp(3, 3, 16, 0.5, (3, 3)))
    return config(64, 32, 1, [latent_layer(1, 4, 2, 8, 4, 2, 50.0, ramp=(2.0, 16, 2.0, 0.5), scale=1.0, mlp=routed_mlp(1, 1, 8, 1.0)),
                              like(tail, 2), tail], logit_scale=3.0)


def _many_streams():
    """Five and more streams take the kernel's form for any number; no rescaled frequencies, no cap, no groups, nothing shared."""
    return config(97, 48, 6, [
        capped_layer(3, 3, 16, 16, 10000.0, 16, scale=0.25, mlp=routed_mlp(4, 4, 24, 50.0)),
        latent_layer(2, 16, 8, 16, 32, 32, 10000.0, scale=0.3, mlp=routed_mlp(6, 1, 64, 1.0, (2, 1), (64, 1.0))),
    ], mult=0.6)


CONFIGS = {"odd_sizes": _odd_sizes(), "wide_heads": _wide_heads(), "smallest": _smallest(), "many_streams": _many_streams()}
PAGES = {"odd_sizes": 4, "wide_heads": 16, "smallest": 2, "many_streams": 8}
# the scale of the random weights: as large as leaves the plain model itself well conditioned
INIT = {name: dict(std=0.15, norm_std=0.3) for name in CONFIGS}
