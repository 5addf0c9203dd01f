"""Fimilix as a list of layers: every layer is a parallel block (one LayerNorm with weight and bias; the mixer and the
feed-forward both read its output and their outputs join the stream together). The mixer is two mixers side by side
whose scaled outputs are added: grouped-query attention without a rotation (a norm per q and k head, a query
temperature that grows with the position, soft-capped scores) and gated linear attention with a decay per key channel.
The feed-forward is a mixture of experts with clipped gates, weighted by a softmax over the chosen experts' logits, or
absent. A span of layers may run several times in a row. The model's final norm is a LayerNorm, the logits are scaled.
The residual stream is 32-bit in either precision. Tensor names are the checkpoint's own: `embed`, `l<i>.norm1(.b)`,
`l<i>.mix.left.{q,k,v,o,q.norm,k.norm}`, `l<i>.mix.right.{q,k,v,g,a1,a2,a2.b,norm,o}`, `l<i>.mlp.router`,
`l<i>.mlp.e<j>.{gate,up,down}`, `final.norm(.b)`, `head`."""

from __future__ import annotations

from ..config.base import register_architecture
from ..config.fimilix import FimilixConfig
from ..parts.base import PartSpec
from .spec import LayerSpec, ModelSpec, ScheduleEntry

# positions enter through the query temperature alone; the cache bounds a request's length
UNBOUNDED_POSITIONS = 1 << 30
GATE_SLOPE = 1.702


def _side_by_side(cfg: FimilixConfig, m: dict) -> PartSpec:
    left, right, q_temp = m["left"], m["right"], m["left"].get("q_temp")
    attention = PartSpec("attention", {
        "hidden": cfg.width, "q_heads": left["heads"], "kv_heads": left["kv_heads"], "head_dim": left["dim"],
        "v_head_dim": left["vdim"], "scale": float(left["scale"]), "softcap": left.get("softcap"),
        "query_temperature": (float(q_temp["coef"]), int(q_temp["every"])) if q_temp else None,
        "qk_norm_eps": cfg.norm_eps, "out_scale": float(m["left_scale"]), "exact_weights": True,
        "q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm"})
    linear = PartSpec("gated_linear_attention", {
        "hidden": cfg.width, "heads": right["heads"], "head_dim": right["dim"], "v_head_dim": right["vdim"],
        "decay_rank": right["decay_rank"], "tau": float(right["tau"]), "norm_eps": cfg.norm_eps,
        "out_scale": float(m["right_scale"]),
        "q": "q", "k": "k", "v": "v", "gate": "g", "a1": "a1", "a2": "a2", "a_bias": "a2.b", "norm": "norm", "o": "o"})
    return PartSpec("side_by_side", {"hidden": cfg.width, "combine": "sum",
                                     "mixers": [(attention, "mix.left.", None), (linear, "mix.right.", None)]})


def _experts(cfg: FimilixConfig, mlp: dict | None) -> PartSpec | None:
    if mlp is None:
        return None
    return PartSpec("routed_experts", {
        "hidden": cfg.width, "experts": mlp["router"]["experts"], "top": mlp["router"]["top"], "inter": mlp["expert"]["ff"],
        "activation": "clipped_swiglu", "limit": float(mlp["expert"]["limit"]), "slope": GATE_SLOPE, "score": "softmax",
        "weight_on": "output", "router": "mlp.router",
        "expert_gate": "mlp.e{}.gate", "expert_up": "mlp.e{}.up", "expert_down": "mlp.e{}.down"})


def fimilix_spec(cfg: FimilixConfig) -> ModelSpec:
    def norm(weight: str, scale: float = 1.0) -> PartSpec:
        return PartSpec("layernorm", {"dim": cfg.width, "eps": cfg.norm_eps, "weight": weight, "bias": weight + ".b",
                                      "out_scale": scale})

    layers = [LayerSpec(PartSpec("parallel", {"input_norm": norm("norm1"), "mixer": _side_by_side(cfg, layer["mixer"]),
                                              "feed_forward": _experts(cfg, layer.get("mlp"))}), f"l{index}.")
              for index, layer in enumerate(cfg.layers)]
    return ModelSpec(
        architecture=cfg.architecture,
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        max_position=UNBOUNDED_POSITIONS,
        embedding="embed",
        final_norm=norm("final.norm", cfg.logit_scale),     # the head is linear: its input scaled is its output scaled
        head="head",
        layers=layers,
        schedule=[ScheduleEntry(index) for index in cfg.layer_runs()],
        residual_dtype="float32",
    )


register_architecture(FimilixConfig.architecture, FimilixConfig.model_type, FimilixConfig, fimilix_spec)
