"""Fimilix without a device: configuration (also the size that is read from a stored tensor), the spec's tensors, parts
and schedule, and what the cache manager makes of side-by-side mixers in layers that run several times."""

import json

import pytest
import torch

import layover_b200 as lb
from fimilix_configs import CONFIGS, config, layer, moe
from layover_b200.cache import CacheManager
from layover_b200.config.base import load_config, resolve_architecture
from layover_b200.models import assemble, spec_for_config
from layover_b200.parts.base import PagedKVNeed, PartSpec, StateNeed, build_part


@pytest.mark.parametrize("name", list(CONFIGS))
def test_config_round_trip_and_registry(name, tmp_path):
    raw = CONFIGS[name]
    cfg = lb.FimilixConfig.from_hf_dict(raw)
    assert lb.FimilixConfig.from_hf_dict(cfg.to_hf_dict()) == cfg
    assert resolve_architecture(raw).config_class is lb.FimilixConfig
    (tmp_path / "config.json").write_text(json.dumps(raw))
    arch, again = load_config(tmp_path)
    assert arch.name == "Fimilix" and again == cfg


def test_the_decay_rank_comes_from_the_stored_tensor_where_the_configuration_leaves_it_out(tmp_path):
    raw = CONFIGS["odd_sizes"]
    folder = lb.write_model_folder(lb.FimilixConfig.from_hf_dict(raw), tmp_path, seed=1)
    stripped = json.loads((folder / "config.json").read_text())
    for entry in stripped["layers"]:
        entry["mixer"]["right"].pop("decay_rank")
    (folder / "config.json").write_text(json.dumps(stripped))
    _, cfg = load_config(folder)
    assert cfg == lb.FimilixConfig.from_hf_dict(raw)
    assert [entry["mixer"]["right"]["decay_rank"] for entry in cfg.layers] == [5, 3, 9]
    with pytest.raises(ValueError, match="decay_rank"):
        lb.FimilixConfig.from_hf_dict(stripped)           # no folder, no shapes


def test_refusals():
    good = CONFIGS["odd_sizes"]
    for change, match in [
        (lambda c: c["layers"][0].update(type="attention"), "unknown type"),
        (lambda c: c["layers"][0]["mixer"]["left"].pop("dim"), "dim"),
        (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "multiple of kv_heads"),
        (lambda c: c["layers"][0]["mixer"]["left"].update(scale=0), "scale"),
        (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=-1.0), "softcap"),
        (lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].update(every=0), "q_temp"),
        (lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].pop("coef"), "q_temp"),
        (lambda c: c["layers"][0]["mixer"]["right"].update(tau=0), "tau"),
        (lambda c: c["layers"][0]["mixer"]["right"].update(heads=0), "heads"),
        (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
        (lambda c: c["layers"][0]["mixer"].update(right_scale="x"), "right_scale"),
        (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "mlp kind"),
        (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "exceeds the experts"),
        (lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0), "limit"),
        (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "ff"),
        (lambda c: c["loop"].update(stop=4), "loop"),
        (lambda c: c["loop"].update(times=0), "loop"),
        (lambda c: c.pop("width"), "lacks"),
    ]:
        raw = json.loads(json.dumps(good))
        change(raw)
        with pytest.raises(ValueError, match=match):
            lb.FimilixConfig.from_hf_dict(raw)


def test_the_specs_tensors_have_the_checkpoints_names_and_shapes():
    raw = config(50, 24, [
        layer((4, 2, 8, 6, 0.3, 5.0, (0.5, 4)), (3, 4, 10, 5, 8.0), (0.5, 2.0), moe(3, 2, 14, 1.5)),
        layer((2, 2, 6, 8, 0.3, None, None), (2, 6, 4, 2, 8.0), (1.0, 1.0)),
    ], loop=(0, 1, 3), logit_scale=0.5)
    spec = spec_for_config(lb.FimilixConfig.from_hf_dict(raw))
    shapes = {s.name: tuple(s.shape) for s in spec.tensor_specs()}
    assert shapes == {
        "embed": (50, 24), "final.norm": (24,), "final.norm.b": (24,), "head": (50, 24),
        "l0.norm1": (24,), "l0.norm1.b": (24,),
        "l0.mix.left.q": (32, 24), "l0.mix.left.k": (16, 24), "l0.mix.left.v": (12, 24), "l0.mix.left.o": (24, 24),
        "l0.mix.left.q.norm": (8,), "l0.mix.left.k.norm": (8,),
        "l0.mix.right.q": (12, 24), "l0.mix.right.k": (12, 24), "l0.mix.right.v": (30, 24), "l0.mix.right.g": (30, 24),
        "l0.mix.right.a1": (5, 24), "l0.mix.right.a2": (12, 5), "l0.mix.right.a2.b": (12,), "l0.mix.right.norm": (10,),
        "l0.mix.right.o": (24, 30),
        "l0.mlp.router": (3, 24), **{f"l0.mlp.e{e}.{n}": (14, 24) for e in range(3) for n in ("gate", "up")},
        **{f"l0.mlp.e{e}.down": (24, 14) for e in range(3)},
        "l1.norm1": (24,), "l1.norm1.b": (24,),
        "l1.mix.left.q": (12, 24), "l1.mix.left.k": (12, 24), "l1.mix.left.v": (16, 24), "l1.mix.left.o": (24, 16),
        "l1.mix.left.q.norm": (6,), "l1.mix.left.k.norm": (6,),
        "l1.mix.right.q": (12, 24), "l1.mix.right.k": (12, 24), "l1.mix.right.v": (8, 24), "l1.mix.right.g": (8, 24),
        "l1.mix.right.a1": (2, 24), "l1.mix.right.a2": (12, 2), "l1.mix.right.a2.b": (12,), "l1.mix.right.norm": (4,),
        "l1.mix.right.o": (24, 8),
    }
    assert spec.residual_dtype == "float32" and not spec.ignorable_tensors
    assert [(e.layer, e.reads_cache_of, e.adds_embedding) for e in spec.schedule] == [(0, None, False)] * 3 + [(1, None, False)]
    kinds = {s.name: s.kind for s in spec.tensor_specs()}
    assert kinds["l0.mlp.router"] == "keep32" and kinds["l0.mix.right.a2.b"] == "vector" and kinds["l0.mix.right.a2"] == "matrix"


@pytest.mark.parametrize("loop, runs", [((1, 3, 2), [0, 1, 2, 1, 2]), ((0, 1, 3), [0, 0, 0, 1, 2]), ((0, 3, 1), [0, 1, 2]),
                                        ((2, 2, 5), [0, 1, 2]), (None, [0, 1, 2])])
def test_looped_layers_run_in_a_row(loop, runs):
    raw = json.loads(json.dumps(CONFIGS["odd_sizes"]))
    raw.pop("loop")
    if loop:
        raw["loop"] = dict(zip(("start", "stop", "times"), loop))
    assert lb.FimilixConfig.from_hf_dict(raw).layer_runs() == runs


def test_every_pass_of_a_looped_layer_has_pages_and_a_state_of_its_own():
    cfg = lb.FimilixConfig.from_hf_dict(CONFIGS["odd_sizes"])
    needs = assemble(spec_for_config(cfg), cfg).cache_needs()
    assert len(needs) == 5 and all(reads is None for _, _, reads in needs)
    assert needs[0][1] == (PagedKVNeed(2, 12, v_head_dim=20), StateNeed((3, 10, 14), torch.float32))
    cache = CacheManager(needs, 64, 4, torch.float32, None, 4)
    assert len(cache.paged) == 3 and len(cache.states) == 3
    assert [len(g.entries) for g in cache.paged] == [1, 2, 2] and [len(g.entries) for g in cache.states] == [1, 2, 2]
    first, second = cache.views[1], cache.views[3]          # layer 1's two passes
    assert first.parts[0].group == second.parts[0].group and first.parts[0].layer != second.parts[0].layer
    assert first.parts[1].group == second.parts[1].group and first.parts[1].layer != second.parts[1].layer
    seq = cache.open("a")
    cache.grow(seq, 70)
    cache.commit(seq, 70)
    assert all(t.first_live == 0 for t in seq.tables)       # every earlier token stays visible: no page goes back
    cache.close(seq)
    cache.check()


def test_part_refusals():
    attention = PartSpec("attention", dict(hidden=16, q_heads=2, kv_heads=1, head_dim=16, q="q", k="k", v="v", o="o"))
    with pytest.raises(ValueError, match="stacked"):        # this attention keeps its own products
        build_part("mixer", PartSpec("side_by_side", {"hidden": 16, "combine": "sum", "mixers": [(attention, "a.", None)]}), "")
    with pytest.raises(ValueError, match="combine"):
        build_part("mixer", PartSpec("side_by_side", {"hidden": 16, "combine": "max", "mixers": [(attention, "a.", None)]}), "")
    experts = dict(hidden=16, experts=4, top=2, inter=8, router="r", expert_gate="g{}", expert_up="u{}", expert_down="d{}", weight_on="output")
    with pytest.raises(ValueError, match="limit"):
        build_part("feed_forward", PartSpec("routed_experts", dict(experts, activation="clipped_swiglu")), "")
    with pytest.raises(ValueError, match="softmax"):
        build_part("feed_forward", PartSpec("routed_experts", dict(experts, score="softmax", renormalize=True)), "")
    with pytest.raises(ValueError, match="query_temperature"):
        build_part("mixer", PartSpec("attention", dict(attention.params, query_temperature=(0.5, 0))), "")
    with pytest.raises(ValueError, match="tau"):
        build_part("mixer", PartSpec("gated_linear_attention", dict(
            hidden=16, heads=2, head_dim=8, v_head_dim=8, decay_rank=4, tau=0.0, norm_eps=1e-5, q="q", k="k", v="v", gate="g", a1="a1",
            a2="a2", a_bias="b", norm="n", o="o")), "")


def test_preset():
    cfg = lb.preset("fimilix-tiny")
    assert isinstance(cfg, lb.FimilixConfig) and cfg.layer_runs() == [0, 1, 1, 2]
    assert spec_for_config(cfg).tensor_specs()
