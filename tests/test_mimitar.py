"""Mimitar without a device: configuration (also the size that is read from a stored tensor), the spec's tensors, parts and
schedule, what the cache manager makes of layers with a token shift and of layers that run with another's tensors, and the
frequencies of the rotations."""

import json

import pytest
import torch

import layover_b200 as lb
import plain_mimitar as plain
from layover_b200.cache import CacheManager
from layover_b200.config.base import load_config, resolve_architecture
from layover_b200.config.mimitar import capped_layer, dense_mlp, latent_layer, routed_mlp
from layover_b200.models import assemble, spec_for_config
from layover_b200.parts.base import PagedKVNeed, PartSpec, Runtime, StateNeed, build_part
from layover_b200.weights.random_init import random_tensor
from mimitar_configs import CONFIGS, config, like


@pytest.mark.parametrize("name", list(CONFIGS))
def test_config_round_trip_and_registry(name, tmp_path):
    raw = CONFIGS[name]
    cfg = lb.MimitarConfig.from_hf_dict(raw)
    assert lb.MimitarConfig.from_hf_dict(cfg.to_hf_dict()) == cfg
    assert resolve_architecture(raw).config_class is lb.MimitarConfig
    (tmp_path / "config.json").write_text(json.dumps(raw))
    arch, again = load_config(tmp_path)
    assert arch.name == "Mimitar" and again == cfg


def test_the_queries_rank_comes_from_the_stored_tensor_where_the_configuration_leaves_it_out(tmp_path):
    raw = CONFIGS["odd_sizes"]
    folder = lb.write_model_folder(lb.MimitarConfig.from_hf_dict(raw), tmp_path, seed=1)
    stripped = json.loads((folder / "config.json").read_text())
    for entry in stripped["layers"]:
        entry["mixer"].pop("q_rank", None)
    (folder / "config.json").write_text(json.dumps(stripped))
    _, cfg = load_config(folder)
    assert cfg == lb.MimitarConfig.from_hf_dict(raw)
    assert [cfg.layers[i]["mixer"]["q_rank"] for i in (0, 2)] == [18, 18]
    with pytest.raises(ValueError, match="q_rank"):
        lb.MimitarConfig.from_hf_dict(stripped)           # no folder, no shapes


def test_refusals():
    for change, match in [
        (lambda c: c["layers"][0].update(type="parallel"), "unknown type"),
        (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
        (lambda c: c["layers"][0]["mixer"].update(rot_dim=8), "rot.dims"),
        (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
        (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("low"), "low"),
        (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=14), "rot.dims"),
        (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=5), "rot.dims"),
        (lambda c: c["layers"][1]["mixer"].pop("rot"), "rot"),
        (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "multiple of kv_heads"),
        (lambda c: c["layers"][1]["mixer"].update(scale=0), "scale"),
        (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
        (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "mlp kind"),
        (lambda c: c["layers"][1]["mlp"].pop("limit"), "limit"),
        (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "exceeds the experts"),
        (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3), "groups"),
        (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=1), "groups"),
        (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "ff"),
        (lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0), "limit"),
        (lambda c: c["layers"][2].update(weights_of=2), "weights_of"),
        (lambda c: c["layers"][2].update(weights_of=1), "not like it"),
        (lambda c: c["layers"][2].update(weights_of=7), "weights_of"),
        (lambda c: c["layers"][0].update(weights_of=2), "leads back"),
        (lambda c: c.update(streams=0), "streams"),
        (lambda c: c.pop("width"), "lacks"),
    ]:
        raw = json.loads(json.dumps(CONFIGS["odd_sizes"]))
        change(raw)
        with pytest.raises(ValueError, match=match):
            lb.MimitarConfig.from_hf_dict(raw)


def test_the_specs_tensors_have_the_checkpoints_names_and_shapes():
    routed = latent_layer(3, 4, 2, 6, 10, 8, 100.0, mlp=routed_mlp(2, 1, 14, 1.5, shared=(12, 2.0)))
    raw = config(50, 24, 2, [routed, capped_layer(4, 2, 8, 6, 100.0, 4, mlp=dense_mlp(20)), like(routed, 0), capped_layer(2, 2, 6, 8, 100.0, 2)])
    spec = spec_for_config(lb.MimitarConfig.from_hf_dict(raw))
    shapes = {s.name: tuple(s.shape) for s in spec.tensor_specs()}

    def hyper(layer, sublayers):
        return {f"l{layer}.hc{q}.{k}": (2, 2) if k == "mix" else (2,) for q in range(1, sublayers + 1) for k in ("in", "out", "mix")}
    assert shapes == {
        "embed": (50, 24), "final.norm": (24,), "head": (50, 24),
        "l0.norm1": (24,), "l0.norm2": (24,), "l0.shift": (24,), **hyper(0, 2),
        "l0.mix.dq": (8, 24), "l0.mix.dq.norm": (8,), "l0.mix.uq": (18, 8), "l0.mix.dkv": (12, 24), "l0.mix.dkv.norm": (10,),
        "l0.mix.uk": (12, 10), "l0.mix.uv": (18, 10), "l0.mix.g": (3, 24), "l0.mix.o": (24, 18),
        "l0.mlp.router": (2, 24), **{f"l0.mlp.e{e}.{n}": (14, 24) for e in range(2) for n in ("gate", "up")},
        **{f"l0.mlp.e{e}.down": (24, 14) for e in range(2)},
        "l0.mlp.shared.gate": (12, 24), "l0.mlp.shared.up": (12, 24), "l0.mlp.shared.down": (24, 12), "l0.mlp.shared.sg": (1, 24),
        "l1.norm1": (24,), "l1.norm2": (24,), "l1.shift": (24,), **hyper(1, 2),
        "l1.mix.q": (32, 24), "l1.mix.k": (16, 24), "l1.mix.v": (12, 24), "l1.mix.o": (24, 24), "l1.mix.q.norm": (32,), "l1.mix.k.norm": (16,),
        "l1.mlp.gate": (20, 24), "l1.mlp.up": (20, 24), "l1.mlp.down": (24, 20),
        "l3.norm1": (24,), "l3.shift": (24,), **hyper(3, 1),
        "l3.mix.q": (12, 24), "l3.mix.k": (12, 24), "l3.mix.v": (16, 24), "l3.mix.o": (24, 16), "l3.mix.q.norm": (12,), "l3.mix.k.norm": (12,),
    }
    assert spec.residual_dtype == "float32" and spec.streams == 2
    assert spec.ignorable_tensors == {"l3.norm2", "l3.hc2.in", "l3.hc2.out", "l3.hc2.mix"}
    assert [(e.layer, e.reads_cache_of) for e in spec.schedule] == [(0, None), (1, None), (0, None), (2, None)]
    kinds = {s.name: s.kind for s in spec.tensor_specs()}
    assert kinds["l0.mlp.router"] == "keep32" and kinds["l0.hc1.mix"] == "vector" and kinds["l0.mix.uq"] == "matrix"


def test_layers_that_share_tensors_have_pages_and_a_state_of_their_own():
    cfg = lb.MimitarConfig.from_hf_dict(CONFIGS["odd_sizes"])
    model = assemble(spec_for_config(cfg), cfg)
    needs = model.cache_needs()
    assert len(model.blocks) == 3 and len(needs) == 4 and all(reads is None for _, _, reads in needs)
    shift = StateNeed((74,), torch.float32)
    assert needs[0][1] == needs[2][1] == (PagedKVNeed(1, 28, values_in_keys=True), shift)
    assert needs[1][1] == (PagedKVNeed(3, 12, v_head_dim=20), shift)
    cache = CacheManager(needs, 64, 4, torch.float32, None, 4)
    assert [len(g.entries) for g in cache.paged] == [2, 1, 1] and [len(g.entries) for g in cache.states] == [4]
    first, again = cache.views[0], cache.views[2]
    assert first.parts[0].group == again.parts[0].group and first.parts[0].layer != again.parts[0].layer
    assert len({view.parts[1].layer for view in cache.views.values()}) == 4
    seq = cache.open("a")
    cache.grow(seq, 70)
    cache.commit(seq, 70)
    assert all(t.first_live == 0 for t in seq.tables)       # every earlier token stays visible: no page goes back
    cache.close(seq)
    cache.check()


def test_a_chain_of_borrowed_layers_and_a_lender_behind_its_borrower():
    cfg = lb.MimitarConfig.from_hf_dict(CONFIGS["wide_heads"])
    assert [cfg.owner(i) for i in range(7)] == [0, 1, 2, 0, 0, 5, 6]
    assert [e.layer for e in spec_for_config(cfg).schedule] == [0, 1, 2, 0, 0, 3, 4]
    cfg = lb.MimitarConfig.from_hf_dict(CONFIGS["smallest"])
    spec = spec_for_config(cfg)
    assert [e.layer for e in spec.schedule] == [0, 1, 1] and spec.layers[1].prefix == "l2."


def _frequencies(kind, params):
    part = build_part("position", PartSpec(kind, params), "")
    part.bind({}, Runtime(torch.float32, torch.device("cpu"), None))
    return part


@pytest.mark.parametrize("rot", [
    {"base": 9000.0, "dims": 6, "scaling": {"factor": 2.5, "low": 1.0, "high": 3.0, "original": 60}},
    {"base": 500000.0, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}},
    {"base": 20.0, "dims": 32, "scaling": {"factor": 3.0, "low": 2.0, "high": 9.0, "original": 33}}, {"base": 100.0, "dims": 2}])
def test_frequencies_by_wavelength_bands(rot):
    part = _frequencies("rotary_half", {"dim": 128, "theta": rot["base"], "rotated": rot["dims"], "band_scaling": rot.get("scaling")})
    assert part.amplitude == 1.0
    torch.testing.assert_close(part.inv_freq().double(), plain.banded_frequencies(rot), rtol=1e-6, atol=0)


@pytest.mark.parametrize("rot", [
    {"base": 3000.0, "dims": 6, "scaling": {"factor": 5.0, "original": 40, "fast": 9.0, "slow": 0.7}},
    {"base": 10000.0, "dims": 64, "scaling": {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0}},
    # the ramp's ends beyond the channels on both sides; a ramp of no width; one frequency
    {"base": 50.0, "dims": 16, "scaling": {"factor": 2.0, "original": 100, "fast": 1000.0, "slow": 0.001}},
    {"base": 10.0, "dims": 32, "scaling": {"factor": 3.0, "original": 4000, "fast": 0.5, "slow": 0.5}},
    {"base": 1000.0, "dims": 2, "scaling": {"factor": 6.0, "original": 64, "fast": 4.0, "slow": 2.0}},
    {"base": 700.0, "dims": 8}])
def test_frequencies_by_a_ramp_over_the_channels(rot):
    part = _frequencies("rotary_pairs", {"dim": rot["dims"], "theta": rot["base"], "rotated": rot["dims"], "ramp_scaling": rot.get("scaling")})
    want, factor = plain.ramped_frequencies(rot)
    torch.testing.assert_close(part.inv_freq().double(), want, rtol=1e-6, atol=0)
    assert abs(part.amplitude - factor) < 1e-12
    if rot.get("scaling") and rot["dims"] == 64:        # the test's own premise: kept, blended and slowed channels
        ratio = want / torch.tensor([rot["base"] ** (-2 * i / 64) for i in range(32)], dtype=torch.float64)
        assert ratio[0] == 1 and abs(ratio[-1] - 1 / 40) < 1e-9 and bool(((ratio > 0.05) & (ratio < 0.95)).any())


def test_part_refusals():
    norm = PartSpec("rmsnorm", {"dim": 16, "eps": 1e-5, "weight": "n"})
    attention = PartSpec("attention", dict(hidden=16, q_heads=2, kv_heads=1, head_dim=16, q="q", k="k", v="v", o="o"))
    names = [{k: f"h{q}.{k}" for k in ("in", "out", "mix")} for q in (1, 2)]
    good = dict(streams=2, hidden=16, connections=names, input_norm=norm, mixer=attention)
    with pytest.raises(ValueError, match="stream"):
        build_part("block", PartSpec("hyper_connected", dict(good, streams=0)), "")
    with pytest.raises(ValueError, match="together"):
        build_part("block", PartSpec("hyper_connected", dict(good, post_norm=norm)), "")
    with pytest.raises(ValueError, match="connections"):
        build_part("block", PartSpec("hyper_connected", dict(good, connections=[])), "")
    with pytest.raises(ValueError, match="ramp"):
        _frequencies("rotary_pairs", {"dim": 8, "theta": 100.0, "ramp_scaling": {"factor": 2.0, "original": 0, "fast": 2.0, "slow": 1.0}})
    latent = dict(hidden=16, heads=2, head_dim=4, rot_dim=4, v_head_dim=4, kv_rank=8, scale=1.0, norm_eps=1e-5, q="q", down="d", down_norm="dn",
                  up_k="k", up_v="v", gate="g", o="o", position=PartSpec("rotary_pairs", {"dim": 4, "theta": 100.0}))
    with pytest.raises(ValueError, match="gate_kind"):
        build_part("mixer", PartSpec("latent_attention", dict(latent, gate_kind="token")), "")
    with pytest.raises(ValueError, match="q_down"):
        build_part("mixer", PartSpec("latent_attention", dict(latent, q_rank=4)), "")
    experts = dict(hidden=16, experts=4, top=2, inter=8, router="r", expert_gate="g{}", expert_up="u{}", expert_down="d{}")
    with pytest.raises(ValueError, match="group_score"):
        build_part("feed_forward", PartSpec("routed_experts", dict(experts, group_score="mean")), "")
    with pytest.raises(ValueError, match="softmax"):
        build_part("feed_forward", PartSpec("routed_experts", dict(experts, score="softmax", groups=2, keep_groups=1)), "")
    build_part("feed_forward", PartSpec("routed_experts", dict(experts, score="softmax_all", groups=2, keep_groups=1, renormalize=True)), "")


def test_random_weights_around_zero_one_and_the_identity():
    spec = spec_for_config(lb.MimitarConfig.from_hf_dict(CONFIGS["many_streams"]))
    made = {s.name: random_tensor(s, 3, 0.02, 0.05) for s in spec.tensor_specs()}
    assert abs(float(made["l0.norm1"].mean())) < 0.05 and abs(float(made["l0.mix.q.norm"].mean()) - 1) < 0.05
    assert (made["l0.hc1.mix"] - torch.eye(6)).abs().max() < 0.3 and abs(float(made["l0.shift"].mean()) - 0.5) < 0.05


def test_preset():
    cfg = lb.preset("mimitar-tiny")
    assert isinstance(cfg, lb.MimitarConfig) and [cfg.owner(i) for i in range(4)] == [0, 1, 1, 3]
    assert spec_for_config(cfg).tensor_specs()
