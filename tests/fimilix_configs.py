"""Small Fimilix configurations for the tests: sizes differ from layer to layer and between the two mixers of a layer,
and values that could hide a fault by being equal (head counts, key and value sizes, the scales of the two mixers) or by
being 1 (experts, chosen experts, a decay rank, `every`, a scale, the laps of a loop) are mixed on purpose."""

from __future__ import annotations


def moe(experts, top, ff, limit):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def layer(left, right, scales, mlp=None):
    """left = (heads, kv_heads, dim, vdim, scale, softcap, (coef, every) or None), right = (heads, dim, vdim, decay rank,
    tau), scales = (left, right)."""
    heads, kv_heads, dim, vdim, scale, softcap, temp = left
    attention = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap:
        attention["softcap"] = softcap
    if temp:
        attention["q_temp"] = {"coef": temp[0], "every": temp[1]}
    linear = dict(zip(("heads", "dim", "vdim", "decay_rank", "tau"), right))
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": attention, "right": linear, "left_scale": scales[0], "right_scale": scales[1]}}


def config(vocab, width, layers, loop=None, logit_scale=None, eps=1e-5):
    raw = {"architecture": "Fimilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        raw["loop"] = dict(zip(("start", "stop", "times"), loop))
    if logit_scale is not None:
        raw["logit_scale"] = logit_scale
    return raw


CONFIGS = {
    # head sizes that are no multiple of 16 or of 4, a row of heads that is no multiple of 8, odd expert widths; a layer
    # without experts inside the loop; the last layer looped too
    "odd_sizes": config(211, 76, [
        layer((6, 2, 12, 20, 0.8, 5.0, (0.6, 7)), (3, 10, 14, 5, 6.0), (0.7, 1.3), moe(7, 3, 40, 1.5)),
        layer((3, 3, 20, 12, 0.5, 3.0, (0.25, 24)), (5, 14, 6, 3, 2.5), (1.2, 0.4)),
        layer((4, 1, 14, 10, 0.9, 8.0, (1.1, 3)), (2, 24, 9, 9, 20.0), (-0.8, 0.6), moe(5, 2, 22, 0.75)),
    ], loop=(1, 3, 2), logit_scale=0.6),
    # head sizes that are multiples of 16: the tensor-core kernels in bfloat16, also the ones for exactly 128 channels;
    # experts of 64 and 128 (the fused epilogue); nine query heads on one key/value head; values wider than keys and keys
    # wider than values; the first layer looped three times
    "wide_heads": config(160, 96, [
        layer((4, 2, 32, 64, 0.4, 6.0, (0.3, 40)), (2, 64, 32, 16, 10.0), (0.9, 0.8), moe(12, 4, 64, 2.5)),
        layer((2, 1, 128, 128, 0.1, 4.0, (0.5, 16)), (1, 128, 96, 24, 8.0), (0.5, 1.1), moe(8, 2, 128, 1.25)),
        layer((9, 1, 48, 16, 0.3, 9.0, (0.7, 100)), (4, 32, 48, 8, 30.0), (1.4, 0.3), moe(6, 5, 48, 3.0)),
    ], loop=(0, 1, 3), logit_scale=1.7),
    # one head, one expert, a rank of 1, a temperature that changes with every token, twenty query heads on one key/value
    # head (more than a tile of the decode kernel holds), all layers looped
    "smallest": config(64, 32, [
        layer((1, 1, 16, 8, 1.0, 2.0, (0.5, 1)), (1, 4, 4, 1, 1.0), (1.0, 1.0), moe(1, 1, 8, 1.0)),
        layer((20, 1, 8, 16, 0.5, 10.0, (2.0, 5)), (2, 4, 20, 2, 3.0), (0.3, 2.0), moe(3, 3, 16, 0.5)),
    ], loop=(0, 2, 2), logit_scale=3.0),
    # no temperature, no cap, no loop, no scales; every expert chosen
    "plain": config(97, 48, [
        layer((3, 3, 16, 16, 0.25, None, None), (3, 16, 16, 8, 12.0), (1.0, 1.0), moe(4, 4, 24, 50.0)),
        layer((2, 1, 32, 16, 0.2, 12.0, None), (2, 160, 16, 4, 5.0), (1.0, 1.0), moe(6, 1, 64, 2.0)),
    ]),
}
PAGES = {"odd_sizes": 4, "wide_heads": 16, "smallest": 2, "plain": 8}
# the scale of the random weights: as large as leaves the plain model itself well conditioned
INIT = {name: dict(std=0.15, norm_std=0.3) for name in CONFIGS}
