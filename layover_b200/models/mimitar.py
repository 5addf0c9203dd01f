"""Mimitar as a list of layers: several residual streams, mixed anew around every sub-layer (hyper-connections), norms with
weights stored around zero before each, a token shift ahead of every mixer. The mixers: grouped-query attention whose q and
k are normed over their whole rows, with a partial rotation by wavelength bands and soft-capped scores, and attention over a
latent whose queries come from a latent of their own, with a ramped rotation of neighbouring channels and a gate per head.
The feed-forward is dense or a mixture of experts, both with clipped gates; the router takes a softmax over all experts,
lets the best groups take part and renormalises, and a shared expert with a gate of its own is added. A layer may run with
another layer's tensors; it then is a second entry of the schedule, with pages and a state of its own. The logits are
scaled. The streams are 32-bit in either precision. Tensor names are the checkpoint's own: `embed`, `l<i>.norm1 / norm2`,
`l<i>.hc1.* / hc2.*` (in, out, mix), `l<i>.shift`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`."""

from __future__ import annotations

from ..config.base import register_architecture
from ..config.mimitar import MimitarConfig
from ..parts.base import PartSpec
from .spec import LayerSpec, ModelSpec, ScheduleEntry

# the rotation's angles are 32-bit products of position and frequency; the cache bounds a request's length
UNBOUNDED_POSITIONS = 1 << 30
GATE_SLOPE = 1.702


def _attention(cfg: MimitarConfig, m: dict) -> PartSpec:
    rot = m["rot"]
    return PartSpec("attention", {
        "hidden": cfg.width, "q_heads": m["heads"], "kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
        "scale": float(m["scale"]), "softcap": m.get("softcap"), "qk_norm": "whole", "qk_norm_eps": cfg.norm_eps, "exact_weights": True,
        "position": PartSpec("rotary_half", {"dim": m["dim"], "theta": float(rot["base"]), "rotated": int(rot["dims"]),
                                             "band_scaling": rot.get("scaling")}),
        "q": "mix.q", "k": "mix.k", "v": "mix.v", "o": "mix.o", "q_norm": "mix.q.norm", "k_norm": "mix.k.norm"})


def _latent(cfg: MimitarConfig, m: dict) -> PartSpec:
    rot = m["rot"]
    return PartSpec("latent_attention", {
        "hidden": cfg.width, "heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"], "v_head_dim": m["vdim"],
        "kv_rank": m["kv_rank"], "q_rank": m["q_rank"], "scale": float(m["scale"]), "norm_eps": cfg.norm_eps, "gate_kind": "head",
        "position": PartSpec("rotary_pairs", {"dim": m["rot_dim"], "theta": float(rot["base"]), "rotated": int(rot["dims"]),
                                              "ramp_scaling": rot.get("scaling")}),
        "q_down": "mix.dq", "q_down_norm": "mix.dq.norm", "q": "mix.uq", "down": "mix.dkv", "down_norm": "mix.dkv.norm",
        "up_k": "mix.uk", "up_v": "mix.uv", "gate": "mix.g", "o": "mix.o"})


def _dense(cfg: MimitarConfig, sizes: dict, prefix: str) -> PartSpec:
    return PartSpec("gated_mlp", {"hidden": cfg.width, "inter": sizes["ff"], "activation": "clipped_swiglu", "limit": float(sizes["limit"]),
                                  "slope": GATE_SLOPE, "gate": prefix + "gate", "up": prefix + "up", "down": prefix + "down"})


def _feed_forward(cfg: MimitarConfig, mlp: dict | None) -> PartSpec | None:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return _dense(cfg, mlp, "mlp.")
    router, shared = mlp["router"], mlp.get("shared")
    groups = router.get("groups") or {}
    return PartSpec("routed_experts", {
        "hidden": cfg.width, "experts": router["experts"], "top": router["top"], "inter": mlp["expert"]["ff"],
        "activation": "clipped_swiglu", "limit": float(mlp["expert"]["limit"]), "slope": GATE_SLOPE,
        "score": "softmax_all", "groups": groups.get("count"), "keep_groups": groups.get("keep"), "group_score": "best",
        "renormalize": True, "weight_on": "output", "router": "mlp.router",
        "expert_gate": "mlp.e{}.gate", "expert_up": "mlp.e{}.up", "expert_down": "mlp.e{}.down",
        "shared": _dense(cfg, shared, "mlp.shared.") if shared else None, "shared_gate": "mlp.shared.sg" if shared else None})


def mimitar_spec(cfg: MimitarConfig) -> ModelSpec:
    def norm(weight: str, scale: float = 1.0) -> PartSpec:
        return PartSpec("rmsnorm", {"dim": cfg.width, "eps": cfg.norm_eps, "weight": weight, "weight_offset": 1.0, "out_scale": scale})

    layers, place, ignorable = [], {}, set()
    for index, layer in enumerate(cfg.layers):
        if cfg.owner(index) != index:
            continue
        mixer = (_attention if layer["type"] == "attention" else _latent)(cfg, layer["mixer"])
        mlp = layer.get("mlp")
        block = PartSpec("hyper_connected", {
            "streams": cfg.streams, "hidden": cfg.width, "mult": cfg.residual_mult, "shift": "shift",
            "connections": [{k: f"hc{q}.{k}" for k in ("in", "out", "mix")} for q in (1, 2)],
            "input_norm": norm("norm1"), "mixer": mixer,
            "post_norm": norm("norm2") if mlp else None, "feed_forward": _feed_forward(cfg, mlp)})
        if not mlp:     # may be stored for every layer; unused where nothing follows the mixer
            ignorable |= {f"l{index}.norm2", *(f"l{index}.hc2.{k}" for k in ("in", "out", "mix"))}
        place[index] = len(layers)
        layers.append(LayerSpec(block, f"l{index}."))
    return ModelSpec(
        architecture=cfg.architecture,
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        max_position=UNBOUNDED_POSITIONS,
        embedding="embed",
        final_norm=norm("final.norm", cfg.logit_scale),     # the head is linear: its input scaled is its output scaled
        head="head",
        layers=layers,
        schedule=[ScheduleEntry(place[cfg.owner(index)]) for index in range(len(cfg.layers))],
        residual_dtype="float32",
        streams=cfg.streams,
        ignorable_tensors=frozenset(ignorable),
    )


register_architecture(MimitarConfig.architecture, MimitarConfig.model_type, MimitarConfig, mimitar_spec)
