"""Typed configuration of Mimitar, read from its own config.json keys.

Mimitar is a decoder with `streams` residual streams instead of one (hyper-connections: every sub-layer reads a weighted
sum of them and all are mixed anew when its output joins, times `residual_mult`) whose layers are listed one by one. Every
layer norms what a sub-layer reads (weights stored around zero), and what a mixer reads is first moved towards what it read
one token before (a token shift). An entry with `weights_of` = j stores nothing: layer j's tensors run once more there,
over other pages and another state.

Kinds of layers (`type`):

"attention": grouped-query attention over every earlier token (`heads`, `kv_heads`, `dim`, `vdim`, `scale`), q and k normed
over their whole rows, a rotation `rot` = {base, dims, scaling} of the first `dims` channels of a head (channels i and i +
dims/2), `scaling` = {factor, low, high, original} by wavelength bands (absent or null: none), and a soft cap `softcap` on
the scores (absent or null: none).

"latent_attention": attention over a latent (`heads`, `dim`, `rot_dim`, `vdim`, `kv_rank`, `scale`) whose queries come from
a latent of `q_rank` channels too, with a gate per head; `rot` = {base, dims = rot_dim, scaling} turns neighbouring channels,
`scaling` = {factor, original, fast, slow} by a ramp over the channels (absent or null: none).

The feed-forward (`mlp`) is {"kind": "dense", ff, limit}, {"kind": "moe", "router": {experts, top, groups}, "expert": {ff,
limit}, "shared": {ff, limit}} (`groups` = {count, keep}, absent or null: none; `shared` absent or null: none) or null.
Sizes that config.json may leave to the stored tensors: `q_rank` (the rows of `l<i>.mix.dq`). Other keys: `vocab`, `width`,
`norm.eps`, `logit_scale` (a factor on the logits). Nothing else is read, and nothing that these keys give stands
anywhere in code.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field

from .kirenex import _need_ints

TYPES = ("attention", "latent_attention")


def _need_positive(where: str, values: dict, names) -> None:
    for name in names:
        value = values.get(name)
        if isinstance(value, bool) or not isinstance(value, (int, float)) or not value > 0:
            raise ValueError(f"{where}.{name} must be a positive number, got {value!r}")


@dataclass(frozen=True)
class MimitarConfig:
    vocab: int
    width: int
    layers: tuple            # of dicts {"type", "mixer", "mlp"[, "weights_of"]}, as config.json lists them
    streams: int = 1
    residual_mult: float = 1.0
    norm_eps: float = 1e-6
    logit_scale: float = 1.0
    eos_token_id: int | None = field(default=None, compare=False)

    architecture = "Mimitar"
    model_type = "mimitar"
    reads_shapes = True

    def __post_init__(self):
        _need_ints("config", {"vocab": self.vocab, "width": self.width, "streams": self.streams}, ("vocab", "width", "streams"))
        if not self.norm_eps > 0:
            raise ValueError("norm.eps must be positive")
        if not self.layers:
            raise ValueError("layers must list at least one layer")
        for index, layer in enumerate(self.layers):
            where, mixer = f"layer {index}", layer.get("mixer") or {}
            if layer.get("type") not in TYPES:
                raise ValueError(f"{where}: unknown type {layer.get('type')!r}; known: {list(TYPES)}")
            if layer["type"] == "attention":
                self._check_attention(where, mixer)
            else:
                self._check_latent(where, mixer)
            if layer.get("mlp") is not None:
                self._check_mlp(where, layer["mlp"])
            owner = layer.get("weights_of")
            if owner is not None:
                if isinstance(owner, bool) or not isinstance(owner, int) or not 0 <= owner < len(self.layers) or owner == index:
                    raise ValueError(f"{where}: weights_of must name another layer, got {owner!r}")
                other = self.layers[owner]
                if any(layer.get(k) != other.get(k) for k in ("type", "mixer", "mlp")):
                    raise ValueError(f"{where}: weights_of names layer {owner}, which is not like it")
        for index in range(len(self.layers)):
            self.owner(index)

    @staticmethod
    def _check_rotation(where: str, rot: dict, most: int, scaling_keys) -> None:
        if not isinstance(rot, dict):
            raise ValueError(f"{where}: mixer.rot is missing")
        _need_positive(where + ": mixer.rot", rot, ("base",))
        _need_ints(where + ": mixer.rot", rot, ("dims",))
        if rot["dims"] % 2 or rot["dims"] > most:
            raise ValueError(f"{where}: mixer.rot.dims must be even and at most {most}, got {rot['dims']}")
        if rot.get("scaling"):
            _need_positive(where + ": mixer.rot.scaling", rot["scaling"], scaling_keys)

    def _check_attention(self, where: str, m: dict) -> None:
        _need_ints(where + ": mixer", m, ("heads", "kv_heads", "dim", "vdim"))
        _need_positive(where + ": mixer", m, ("scale",))
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"{where}: mixer.heads ({m['heads']}) must be a multiple of kv_heads ({m['kv_heads']})")
        if m.get("softcap") is not None:
            _need_positive(where + ": mixer", m, ("softcap",))
        self._check_rotation(where, m.get("rot"), m["dim"], ("factor", "low", "high", "original"))

    def _check_latent(self, where: str, m: dict) -> None:
        _need_ints(where + ": mixer", m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
        _need_positive(where + ": mixer", m, ("scale",))
        self._check_rotation(where, m.get("rot"), m["rot_dim"], ("factor", "original", "fast", "slow"))
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError(f"{where}: mixer.rot.dims ({m['rot']['dims']}) must be rot_dim ({m['rot_dim']})")

    @staticmethod
    def _check_mlp(where: str, mlp: dict) -> None:
        if mlp.get("kind") == "dense":
            _need_ints(where + ": mlp", mlp, ("ff",))
            _need_positive(where + ": mlp", mlp, ("limit",))
            return
        if mlp.get("kind") != "moe":
            raise ValueError(f"{where}: unknown mlp kind {mlp.get('kind')!r}; known: ['dense', 'moe']")
        router = mlp.get("router") or {}
        _need_ints(where + ": mlp.router", router, ("experts", "top"))
        for name in ("expert", "shared"):
            if name == "expert" or mlp.get(name) is not None:
                _need_ints(f"{where}: mlp.{name}", mlp.get(name) or {}, ("ff",))
                _need_positive(f"{where}: mlp.{name}", mlp.get(name) or {}, ("limit",))
        if router["top"] > router["experts"]:
            raise ValueError(f"{where}: mlp.router.top ({router['top']}) exceeds the experts ({router['experts']})")
        groups = router.get("groups")
        if groups:
            _need_ints(where + ": mlp.router.groups", groups, ("count", "keep"))
            if (router["experts"] % groups["count"] or groups["keep"] > groups["count"]
                    or groups["keep"] * (router["experts"] // groups["count"]) < router["top"]):
                raise ValueError(f"{where}: mlp.router.groups {groups!r} cannot give a token {router['top']} of {router['experts']} experts")

    def owner(self, index: int) -> int:
        """The layer whose tensors layer `index` runs with."""
        seen = set()
        while self.layers[index].get("weights_of") is not None:
            if index in seen:
                raise ValueError(f"layer {index}: weights_of leads back to it")
            seen.add(index)
            index = self.layers[index]["weights_of"]
        return index

    @classmethod
    def from_hf_dict(cls, raw: dict, shapes: dict | None = None) -> "MimitarConfig":
        """`shapes` (tensor name -> shape of the stored tensors) fills in what config.json leaves to them: the size of the
        queries' latent."""
        missing = [k for k in ("vocab", "width", "layers") if k not in raw]
        if missing:
            raise ValueError(f"config.json lacks {missing}")
        layers = tuple(copy.deepcopy(layer) for layer in raw["layers"])
        for index, layer in enumerate(layers):
            mixer = layer.get("mixer")
            if layer.get("type") == "latent_attention" and isinstance(mixer, dict) and "q_rank" not in mixer:
                at = layer.get("weights_of")
                shape = (shapes or {}).get(f"l{index if at is None else at}.mix.dq")
                if shape is None:
                    raise ValueError(f"layer {index}: mixer.q_rank is neither in config.json nor given by a stored l{index}.mix.dq")
                mixer["q_rank"] = int(shape[0])
        eos = raw.get("eos_token_id")
        return cls(
            vocab=raw["vocab"], width=raw["width"], layers=layers, streams=raw.get("streams", 1),
            residual_mult=float(raw.get("residual_mult", 1.0)),
            norm_eps=float((raw.get("norm") or {}).get("eps", 1e-6)),
            logit_scale=float(raw.get("logit_scale", 1.0)),
            eos_token_id=eos[0] if isinstance(eos, list) else eos,
        )

    def to_hf_dict(self) -> dict:
        """The config.json that reads back as this configuration."""
        return {
            "architecture": self.architecture,
            "layers": [copy.deepcopy(layer) for layer in self.layers],
            "logit_scale": self.logit_scale,
            "norm": {"eps": self.norm_eps},
            "residual_mult": self.residual_mult,
            "streams": self.streams,
            "vocab": self.vocab,
            "width": self.width,
        }


def capped_layer(heads, kv_heads, dim, vdim, base, rotated, bands=None, softcap=None, scale=None, mlp=None) -> dict:
    """One `attention` entry of `layers`; bands = (factor, low, high, original)."""
    rot = {"base": base, "dims": rotated}
    if bands:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), bands))
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5, "rot": rot}
    if softcap:
        mixer["softcap"] = softcap
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def latent_layer(heads, dim, rot_dim, vdim, kv_rank, q_rank, base, ramp=None, scale=None, mlp=None) -> dict:
    """One `latent_attention` entry of `layers`; ramp = (factor, original, fast, slow)."""
    rot = {"base": base, "dims": rot_dim}
    if ramp:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), ramp))
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": rot}}


def dense_mlp(ff, limit=7.0) -> dict:
    return {"kind": "dense", "ff": ff, "limit": limit}


def routed_mlp(experts, top, ff, limit=7.0, groups=None, shared=None) -> dict:
    """groups = (count, keep), shared = (ff, limit)."""
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = dict(zip(("count", "keep"), groups))
    out = {"kind": "moe", "router": router, "expert": {"ff": ff, "limit": limit}}
    if shared:
        out["shared"] = dict(zip(("ff", "limit"), shared))
    return out


# Named shapes for the command line and the benchmark (inputs, like a parsed config.json).
MIMITAR_PRESETS: dict[str, dict] = {
    "mimitar-tiny": dict(
        vocab=336, width=104, streams=3, residual_mult=0.4, norm_eps=1e-5, logit_scale=0.7,
        layers=(latent_layer(4, 16, 12, 24, 40, 28, 20000.0, ramp=(6.0, 128, 16.0, 2.0), mlp=routed_mlp(8, 2, 48, 3.0, (4, 2), (40, 2.5))),
                capped_layer(4, 2, 32, 24, 60000.0, 20, bands=(3.0, 1.0, 4.0, 96), softcap=20.0, mlp=dense_mlp(160, 3.0)),
                dict(capped_layer(4, 2, 32, 24, 60000.0, 20, bands=(3.0, 1.0, 4.0, 96), softcap=20.0, mlp=dense_mlp(160, 3.0)), weights_of=1),
                latent_layer(2, 24, 8, 16, 48, 32, 20000.0))),
}
