"""Typed configuration of Fimilix, read from its own config.json keys.

Fimilix is a decoder whose layers are listed one by one. Every layer is a parallel block: one LayerNorm (weight and
bias), and the mixer and the feed-forward both read its output. `loop` = `{start, stop, times}` runs layers start ..
stop-1 `times` times in a row with the same weights (each pass keeps a cache and a state of its own). The one kind of
layer (`type`: "parallel") mixes with two mixers side by side, `left_scale` * left + `right_scale` * right:

`left`: grouped-query attention over every earlier token (`heads`, `kv_heads`, `dim`, `vdim`, `scale`) without a
rotation, an RMS norm per q and k head, a query temperature `q_temp` = {coef, every} that grows with the position
(absent or null: none) and a soft cap `softcap` on the scores (absent or null: none).

`right`: gated linear attention (`heads`, `dim`, `vdim`) with a decay per key channel, the `tau`-th root of a sigmoid
gate. The rank of the gate's two small matrices is the one size that config.json may leave to the stored tensors
(`decay_rank`, else the rows of `l<i>.mix.right.a1`).

The feed-forward (`mlp`) is `{"kind": "moe", "router": {experts, top}, "expert": {ff, limit}}` (a mixture of experts
with clipped gates; weights by softmax over the chosen experts' logits) or null. Other keys: `vocab`, `width`,
`norm.eps`, `logit_scale` (a factor on the logits). Nothing else is read, and nothing that these keys give stands
anywhere in code.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field

from .kirenex import _need_ints, _positive_int


@dataclass(frozen=True)
class FimilixConfig:
    vocab: int
    width: int
    layers: tuple            # of dicts {"type", "mixer", "mlp"}, as config.json lists them
    norm_eps: float = 1e-6
    logit_scale: float = 1.0
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    eos_token_id: int | None = field(default=None, compare=False)

    architecture = "Fimilix"
    model_type = "fimilix"
    reads_shapes = True

    def __post_init__(self):
        _need_ints("config", {"vocab": self.vocab, "width": self.width}, ("vocab", "width"))
        if not self.norm_eps > 0:
            raise ValueError("norm.eps must be positive")
        if not self.layers:
            raise ValueError("layers must list at least one layer")
        for index, layer in enumerate(self.layers):
            where, mixer = f"layer {index}", layer.get("mixer") or {}
            if layer.get("type") != "parallel":
                raise ValueError(f"{where}: unknown type {layer.get('type')!r}; known: ['parallel']")
            left, right = mixer.get("left") or {}, mixer.get("right") or {}
            _need_ints(where + ": mixer.left", left, ("heads", "kv_heads", "dim", "vdim"))
            _need_ints(where + ": mixer.right", right, ("heads", "dim", "vdim", "decay_rank"))
            if left["heads"] % left["kv_heads"]:
                raise ValueError(f"{where}: left.heads ({left['heads']}) must be a multiple of kv_heads ({left['kv_heads']})")
            for key in ("left_scale", "right_scale"):
                if isinstance(mixer.get(key), bool) or not isinstance(mixer.get(key), (int, float)):
                    raise ValueError(f"{where}: mixer.{key} must be a number, got {mixer.get(key)!r}")
            if not float(left.get("scale") or 0) > 0:
                raise ValueError(f"{where}: mixer.left.scale must be positive")
            if left.get("softcap") is not None and not float(left["softcap"]) > 0:
                raise ValueError(f"{where}: mixer.left.softcap must be positive")
            q_temp = left.get("q_temp")
            if q_temp is not None and (not _positive_int(q_temp.get("every")) or q_temp.get("coef") is None):
                raise ValueError(f"{where}: mixer.left.q_temp needs a coef and a positive integer every, got {q_temp!r}")
            if not float(right.get("tau") or 0) > 0:
                raise ValueError(f"{where}: mixer.right.tau must be positive")
            mlp = layer.get("mlp")
            if mlp is not None:
                if mlp.get("kind") != "moe":
                    raise ValueError(f"{where}: unknown mlp kind {mlp.get('kind')!r}; known: ['moe']")
                router, expert = mlp.get("router") or {}, mlp.get("expert") or {}
                _need_ints(where + ": mlp.router", router, ("experts", "top"))
                _need_ints(where + ": mlp.expert", expert, ("ff",))
                if router["top"] > router["experts"]:
                    raise ValueError(f"{where}: mlp.router.top ({router['top']}) exceeds the experts ({router['experts']})")
                if not float(expert.get("limit") or 0) > 0:
                    raise ValueError(f"{where}: mlp.expert.limit must be positive")
        if not (0 <= self.loop_start <= self.loop_stop <= len(self.layers)) or self.loop_times < 1:
            raise ValueError(f"loop {self.loop_start}..{self.loop_stop} x {self.loop_times} does not fit {len(self.layers)} layers")

    @classmethod
    def from_hf_dict(cls, raw: dict, shapes: dict | None = None) -> "FimilixConfig":
        """`shapes` (tensor name -> shape of the stored tensors) fills in what config.json leaves to them: the rank of a
        layer's decay matrices."""
        missing = [k for k in ("vocab", "width", "layers") if k not in raw]
        if missing:
            raise ValueError(f"config.json lacks {missing}")
        layers = tuple(copy.deepcopy(layer) for layer in raw["layers"])
        for index, layer in enumerate(layers):
            right = (layer.get("mixer") or {}).get("right")
            if isinstance(right, dict) and "decay_rank" not in right:
                shape = (shapes or {}).get(f"l{index}.mix.right.a1")
                if shape is None:
                    raise ValueError(f"layer {index}: mixer.right.decay_rank is neither in config.json nor given by a stored "
                                     f"l{index}.mix.right.a1")
                right["decay_rank"] = int(shape[0])
        loop, eos = raw.get("loop") or {}, raw.get("eos_token_id")
        return cls(
            vocab=raw["vocab"], width=raw["width"], layers=layers,
            norm_eps=float((raw.get("norm") or {}).get("eps", 1e-6)),
            logit_scale=float(raw.get("logit_scale", 1.0)),
            loop_start=int(loop.get("start", 0)), loop_stop=int(loop.get("stop", 0)), loop_times=int(loop.get("times", 1)),
            eos_token_id=eos[0] if isinstance(eos, list) else eos,
        )

    def to_hf_dict(self) -> dict:
        """The config.json that reads back as this configuration."""
        return {
            "architecture": self.architecture,
            "layers": [copy.deepcopy(layer) for layer in self.layers],
            "logit_scale": self.logit_scale,
            "loop": {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times},
            "norm": {"eps": self.norm_eps},
            "vocab": self.vocab,
            "width": self.width,
        }

    def layer_runs(self) -> list[int]:
        """The layers in running order: the looped ones `loop_times` times in a row."""
        span = list(range(self.loop_start, self.loop_stop))
        return list(range(self.loop_start)) + span * self.loop_times + list(range(self.loop_stop, len(self.layers)))


def gated_parallel_layer(heads, kv_heads, dim, vdim, linear_heads, linear_dim, linear_vdim, decay_rank, tau=12.0, scale=None,
                         softcap=None, q_temp=None, left_scale=1.0, right_scale=1.0, experts=None, top=1, ff=None, limit=7.0) -> dict:
    """One `parallel` entry of `layers`; q_temp = (coef, every)."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if softcap:
        left["softcap"] = softcap
    if q_temp:
        left["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    right = {"heads": linear_heads, "dim": linear_dim, "vdim": linear_vdim, "decay_rank": decay_rank, "tau": tau}
    return {"type": "parallel",
            "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale},
            "mlp": {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}} if experts else None}


# Named shapes for the command line and the benchmark (inputs, like a parsed config.json).
FIMILIX_PRESETS: dict[str, dict] = {
    "fimilix-tiny": dict(
        vocab=336, width=104, norm_eps=1e-5, logit_scale=0.5, loop_start=1, loop_stop=2, loop_times=2,
        layers=(gated_parallel_layer(4, 2, 32, 24, 3, 16, 40, 8, tau=8.0, softcap=20.0, q_temp=(0.3, 20), left_scale=0.7,
                                     right_scale=1.1, experts=8, top=2, ff=48, limit=3.0),
                gated_parallel_layer(2, 1, 16, 48, 4, 24, 16, 12, softcap=15.0, q_temp=(0.4, 50), left_scale=0.8,
                                     right_scale=0.5, experts=6, top=3, ff=64, limit=2.5),
                gated_parallel_layer(3, 3, 48, 32, 2, 32, 32, 4, tau=4.0, q_temp=(0.2, 33), softcap=40.0))),
}
