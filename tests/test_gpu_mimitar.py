"""Mimitar on the GPU against the plain implementation: every mechanism alone, then whole models in every way a
request can be cut, batched and decoded, in 32-bit and in bfloat16."""

import json

import numpy as np
import pytest
import torch

import layover_b200 as lb
import plain_mimitar as plain
from conftest import random_prompt, tolerance
from layover_b200 import ops
from layover_b200.cache import CacheManager
from layover_b200.config.mimitar import capped_layer, dense_mlp, latent_layer
from layover_b200.engine.batch import BatchBuilder, StepEntry
from layover_b200.parts.base import Part, PartSpec, build_part, register_mixer, unregister, walk_parts
from layover_b200.parts.norm import StreamUpdate
from mimitar_configs import CONFIGS, INIT, PAGES, config
from replay_helpers import collect, max_live_tokens, mixed, portions, run_trace, tail_decoded
from test_gpu_fimilix import (CUTS, DTYPES, F, _names, _uneven, bound_part, close, compare, cuts_of, in_company, mixer_harness,
                              random_tensors, run_cuts, stored_as)

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------ residual streams
STREAM_SHAPES = [(1, 40), (2, 36), (2, 1024), (3, 74), (3, 512), (4, 2048), (5, 100), (7, 33), (2, 4100), (4, 8192), (1, 4091), (16, 64)]


def stream_case(streams, width, tokens, dtype, seed=0):
    gen = torch.Generator().manual_seed(seed + streams * 1000 + width)
    x = torch.randn(tokens, streams, width, generator=gen) * 2
    y = torch.randn(tokens, width, generator=gen).to(dtype)
    mix = torch.eye(streams) + 0.4 * torch.randn(streams, streams, generator=gen)
    gain, read = torch.randn(streams, generator=gen), torch.randn(streams, generator=gen) + 0.5
    weight, mu = 1 + 0.3 * torch.randn(width, generator=gen), torch.rand(width, generator=gen) * 1.4 - 0.2
    return x, y, mix, gain, read, weight, mu


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("streams, width", STREAM_SHAPES)
def test_streams_are_mixed_read_and_normed(dtype, streams, width):
    """All streams from the old ones at once (the mix is far from symmetric), read as a weighted sum, normed; nothing
    pending; equal streams that are one row; picked rows with the plain sum."""
    tokens, eps = 9, 1e-3
    x, y, mix, gain, read, weight, _ = stream_case(streams, width, tokens, dtype)
    dev = [t.cuda() for t in (x, y, mix, gain, read, weight)]
    made = plain.write_streams(x.to(F), mix.to(F), gain.to(F), y.to(F))
    want = plain.rms_norm(plain.read_streams(made, read.to(F)), weight.to(F), eps)
    out, x_out = torch.empty(tokens, width, dtype=dtype, device="cuda"), torch.empty_like(dev[0])
    before = dev[0].clone()
    ops.stream_norm(dev[0], (dev[1], dev[2], dev[3]), dev[4], dev[5], eps, out, x_out)
    assert torch.equal(before, dev[0])
    close(x_out, made, torch.float32, "streams")
    close(out, want, dtype, "normed sum")
    # nothing pending, and the streams as one row
    row = x[:, :1].cuda().expand(-1, streams, -1)
    ops.stream_norm(row, None, dev[4], dev[5], eps, out)
    close(out, plain.rms_norm(x[:, 0].to(F) * read.to(F).sum(), weight.to(F), eps), dtype, "equal streams")
    ops.stream_norm(row, (dev[1], dev[2], dev[3]), dev[4], dev[5], eps, out, x_out)
    close(x_out, plain.write_streams(x[:, :1].to(F).expand(-1, streams, -1), mix.to(F), gain.to(F), y.to(F)), torch.float32, "from equal streams")
    # picked rows of the plain sum
    rows = torch.tensor([8, 0, 3], dtype=torch.int32, device="cuda")
    picked = torch.empty(3, width, dtype=dtype, device="cuda")
    ops.stream_norm(dev[0], (dev[1], dev[2], dev[3]), None, dev[5], eps, picked, rows=rows)
    close(picked, plain.rms_norm(made.sum(dim=1), weight.to(F), eps)[[8, 0, 3]], dtype, "picked rows")


def test_stream_refusals():
    x = torch.randn(3, 2, 16, device="cuda")
    w, out = torch.ones(16, device="cuda"), torch.empty(3, 16, device="cuda")
    update = (torch.randn(3, 16, device="cuda"), torch.eye(2, device="cuda"), torch.ones(2, device="cuda"))
    with pytest.raises(ValueError, match="another"):
        ops.stream_norm(x, update, None, w, 1e-5, out, x)
    with pytest.raises(ValueError, match="read"):
        ops.stream_norm(x, update, torch.ones(3, device="cuda"), w, 1e-5, out)
    with pytest.raises(ValueError, match="update"):
        ops.stream_norm(x, (update[0], torch.eye(3, device="cuda"), update[2]), None, w, 1e-5, out)
    wide = torch.randn(1, 2, 8196, device="cuda")
    with pytest.raises(ValueError, match="size"):
        ops.stream_norm(wide, None, None, torch.ones(8196, device="cuda"), 1e-5, torch.empty(1, 8196, device="cuda"))


class _Probe(Part):
    """A mixer that hands on what it read, so that a test can see it."""

    def __init__(self, params, prefix):
        super().__init__(params, prefix)

    def cache_need(self):
        return None

    def forward(self, h, batch, cache):
        assert cache is None
        return h.clone()


@pytest.fixture
def probe():
    register_mixer("probe", _Probe)
    yield
    unregister("mixer", "probe")


def block_spec(streams, width, mult=0.7, eps=1e-5):
    return PartSpec("hyper_connected", {
        "streams": streams, "hidden": width, "mult": mult, "shift": "shift", "connections": [{k: f"hc1.{k}" for k in ("in", "out", "mix")}],
        "input_norm": PartSpec("rmsnorm", {"dim": width, "eps": eps, "weight": "norm1", "weight_offset": 1.0}), "mixer": PartSpec("probe", {})})


def block_harness(spec, tensors, dtype, slots=3):
    part = bound_part("block", spec, tensors, dtype)
    cache = CacheManager([(0, part.cache_need(), None)], 1, 16, dtype, "cuda", slots, ops.RECORD_WORDS)
    builder = BatchBuilder(cache, torch.device("cuda"), tuple(s for p in walk_parts(part) for s in p.tile_sizes(dtype)))

    def step(entries, update):      # [(sequence, x rows, y rows)] -> (what the mixer read, the streams), per entry
        made = [StepEntry(seq, [0] * x.shape[0], []) for seq, x, _ in entries]
        batch = builder.build(made)
        x = torch.cat([x for _, x, _ in entries]).cuda()
        y = torch.cat([y for _, _, y in entries]).to(dtype).cuda()
        streams, out = part.forward(x, StreamUpdate(y, *update), batch, cache.view(0))
        for entry in made:
            cache.commit(entry.seq, entry.seq.num_tokens + len(entry.tokens))
        sizes = [x.shape[0] for _, x, _ in entries]
        return [(h, s) for h, s in zip(torch.split(out.value.float().cpu(), sizes), torch.split(streams.cpu(), sizes))], out
    return part, cache, step


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("streams, width", [(2, 64), (3, 74), (1, 40), (6, 48), (4, 1100), (2, 2560)])
def test_token_shift_in_every_cut(probe, dtype, streams, width):
    """What the mixer reads mixes with what it read one token before, unshifted, whichever step brought that token; the
    same bits whatever the cut; requests beside one another; slots that are used again start from zeros."""
    spec, eps, n = block_spec(streams, width), 1e-5, 43
    x, y, mix, gain, read, weight, mu = stream_case(streams, width, n, dtype, seed=5)
    tensors = {"norm1": (weight - 1).to(torch.bfloat16).float(), "shift": mu.to(torch.bfloat16).float(),
               "hc1.in": read.to(torch.bfloat16).float(), "hc1.out": gain.to(torch.bfloat16).float(), "hc1.mix": mix.to(torch.bfloat16).float()}
    part, cache, step = block_harness(spec, tensors, dtype)
    update = (mix.cuda(), gain.cuda())
    t = {k: v.to(F) for k, v in tensors.items()}

    def reference(x, y):
        made = plain.write_streams(x.to(F), mix.to(F), gain.to(F), y.to(F))
        return plain.shift(plain.rms_norm(plain.read_streams(made, t["hc1.in"]), 1 + t["norm1"], eps), t["shift"]), made
    want, streams_want = reference(x, y)
    first = None
    for name, cuts in cuts_of(n).items():
        seq, at, got = cache.open(f"s{next(_names)}"), 0, []
        for count in cuts:
            (rows,), pending = step([(seq, x[at:at + count], y[at:at + count])], update)
            got.append(rows)
            at += count
        cache.close(seq)
        h, s = torch.cat([g[0] for g in got]), torch.cat([g[1] for g in got])
        close(h, want, dtype, name)
        close(s, streams_want, torch.float32, name + ": streams")
        first = h if first is None else first
        assert torch.equal(first, h), name
        assert torch.allclose(pending.gain.cpu(), 0.7 * tensors["hc1.out"]) and torch.equal(pending.mix.cpu(), tensors["hc1.mix"])
    # two requests with different rows at a time; one joins, ends and its slot goes to the next
    flipped = reference(x.flip(0), y.flip(0))[0]
    for _ in range(2):
        a, b = cache.open("a"), cache.open("b")
        one, _ = step([(a, x[:11], y[:11])], update)
        two, _ = step([(a, x[11:12], y[11:12]), (b, x.flip(0)[:6], y.flip(0)[:6])], update)
        three, _ = step([(b, x.flip(0)[6:7], y.flip(0)[6:7]), (a, x[12:], y[12:])], update)
        close(torch.cat((one[0][0], two[0][0], three[1][0])), want, dtype, "a beside b")
        close(torch.cat((two[1][0], three[0][0])), flipped[:7], dtype, "b beside a")
        cache.close(b); cache.close(a)
    # the first token mixes with zeros, not with what the slot's last owner left
    close(first[0], want[0], dtype)
    assert (want[0] - plain.rms_norm(plain.read_streams(streams_want, t["hc1.in"]), 1 + t["norm1"], eps)[0]).abs().max() > 0.05


# ------------------------------------------------------------------ rotations
@pytest.mark.parametrize("kind, scaling", [("rotary_half", {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 256}), ("rotary_half", None),
                                           ("rotary_pairs", {"factor": 12.0, "original": 256, "fast": 20.0, "slow": 0.8}), ("rotary_pairs", None)])
def test_the_steps_table_of_cosines_and_sines(kind, scaling):
    import types

    rot = {"base": 30000.0, "dims": 24, "scaling": scaling}
    part = bound_part("position", PartSpec(kind, {"dim": 24, "theta": rot["base"], "rotated": 24,
                                                  "band_scaling" if kind == "rotary_half" else "ramp_scaling": scaling}), {}, torch.float32)
    freq, factor = (plain.banded_frequencies(rot), 1.0) if kind == "rotary_half" else plain.ramped_frequencies(rot)
    assert (factor != 1.0) == (kind == "rotary_pairs" and scaling is not None)
    positions = torch.tensor([0, 1, 7, 255, 256, 1000, 4095], dtype=torch.int32, device="cuda")
    batch = types.SimpleNamespace(positions=positions, n_tokens=positions.numel(), shared={})
    table = part.tables(batch)
    assert part.tables(batch) is table
    angles = positions.cpu().to(F)[:, None] * freq
    want = factor * torch.stack((angles.cos(), angles.sin()), dim=1)
    assert (table.cpu().to(F) - want).abs().max() < 5e-4       # a 32-bit angle of thousands


# ------------------------------------------------------------------ attention with whole-row norms and capped scores
def attention_spec(hidden, m):
    rot = m["rot"]
    return PartSpec("attention", dict(
        hidden=hidden, q_heads=m["heads"], kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"], scale=m["scale"], softcap=m.get("softcap"),
        qk_norm="whole", qk_norm_eps=1e-5, exact_weights=True, q="q", k="k", v="v", o="o", q_norm="q.norm", k_norm="k.norm",
        position=PartSpec("rotary_half", {"dim": m["dim"], "theta": rot["base"], "rotated": rot["dims"], "band_scaling": rot.get("scaling")})))


def attention(heads, kv, d, e, scale, cap, base, dims, bands=None):
    rot = {"base": base, "dims": dims}
    if bands:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), bands))
    return {"heads": heads, "kv_heads": kv, "dim": d, "vdim": e, "scale": scale, "softcap": cap, "rot": rot}


ATTENTION_SHAPES = [  # hidden, mixer, page
    (40, attention(6, 3, 12, 20, 0.6, 4.0, 9000.0, 6, (2.5, 1.0, 3.0, 60)), 4),
    (64, attention(4, 2, 32, 64, 0.4, 6.0, 20000.0, 16, (6.0, 1.0, 4.0, 120)), 16),
    (64, attention(2, 1, 128, 128, 0.1, 3.0, 10000.0, 128), 16), (32, attention(20, 1, 8, 16, 0.5, 10.0, 100.0, 2), 2),
    (48, attention(3, 3, 16, 16, 0.6, None, 500.0, 16, (3.0, 1.0, 8.0, 50)), 8), (48, attention(9, 1, 48, 16, 0.3, 2.0, 10000.0, 46), 16),
    (56, attention(2, 2, 160, 96, 0.1, 5.0, 10000.0, 64), 8), (38, attention(40, 5, 14, 10, 0.7, 5.0, 700.0, 14), 4)]


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("shape", ATTENTION_SHAPES)
def test_attention_in_every_cut(dtype, shape):
    hidden, m, page = shape
    spec = attention_spec(hidden, m)
    tensors = random_tensors(build_part("mixer", spec, "").tensor_specs(), seed=m["dim"] + m["vdim"])
    part, cache, step = mixer_harness(spec, tensors, dtype, page_tokens=page, pages=120)
    n = 90
    rows = (torch.randn(n, hidden, generator=torch.Generator().manual_seed(5)) * 1.5).to(dtype).float()
    want = plain.attention_mixer(rows.to(F), stored_as(tensors, dtype), m, 1e-5)
    for name, cuts in cuts_of(n).items():
        close(run_cuts(cache, step, rows, cuts), want, dtype, name, slack=3)
    in_company(cache, step, rows, want, dtype, 3)


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
def test_a_norm_over_all_heads_is_not_a_norm_per_head(dtype):
    """One head ten times the size of the others: normed over the whole row it keeps that ratio, and the others stay small."""
    heads, kv, d, hidden = 4, 2, 16, 128
    m = attention(heads, kv, d, d, 1.0, None, 10000.0, 2)
    tensors = random_tensors(build_part("mixer", attention_spec(hidden, m), "").tensor_specs(), seed=4)
    part, cache, step = mixer_harness(attention_spec(hidden, m), tensors, dtype)
    seq = cache.open("s")
    cache.grow(seq, 6)
    builder = BatchBuilder(cache, torch.device("cuda"), part.tile_sizes(dtype))
    batch = builder.build([StepEntry(seq, [0] * 6, [])])
    proj = torch.randn(6, (heads + 2 * kv) * d, generator=torch.Generator().manual_seed(1))
    proj[:, 2 * d: 3 * d] *= 10
    proj[:, heads * d: heads * d + d] *= 10
    q = torch.empty(6, heads * d, dtype=dtype, device="cuda")
    view = cache.view(0)
    w_q, w_k = tensors["q.norm"].cuda(), tensors["k.norm"].cuda()
    ops.heads_bias_rope_kv(proj.cuda(), q, view.k_pool, view.v_pool, None, None, None, None, batch.groups[0].slot_map, None, 0, None, heads, kv, d, d,
                           4, w_q, w_k, 1e-5, whole_norm=True)
    want = plain.rms_norm(proj[:, : heads * d].to(F), tensors["q.norm"].to(F), 1e-5)
    close(q, want, dtype, "q")
    k = torch.stack([view.k_pool[int(s) // 4, :, int(s) % 4] for s in batch.groups[0].slot_map.cpu()])
    close(k.reshape(6, kv * d), plain.rms_norm(proj[:, heads * d: (heads + kv) * d].to(F), tensors["k.norm"].to(F), 1e-5), dtype, "k")
    sizes = want.view(6, heads, d).pow(2).mean(dim=2).sqrt().mean(dim=0)
    assert sizes[2] > 4 * sizes[0]                  # the test's own premise
    with pytest.raises(ValueError, match="q_norm_w"):
        ops.heads_bias_rope_kv(proj.cuda(), q, view.k_pool, view.v_pool, None, None, None, None, batch.groups[0].slot_map, None, 0, None, heads, kv,
                               d, d, 4, w_q, w_k, 1e-5)


def places_in(n, page):
    last = n - 1
    return sorted({0, 1, page - 1, page, 31, 64, 65, last // page * page, last // page * page - 1, last - 1, last})


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("d, e, page", [(16, 16, 4), (64, 32, 16), (128, 128, 16), (12, 20, 4)])
def test_one_key_among_hundreds(dtype, d, e, page):
    """The last query looks for ONE key, at the first position, at page and tile borders, far back and next to it. The pair's
    channels are not turned (the first two are, and they are zero), so that its score stands out whatever the distance."""
    hidden, n, scale, cap = max(3 * d + e + 4, 2 * e), 330, 8.0 / d ** 0.5, 11.0
    m = attention(2, 1, d, e, scale, cap, 10000.0, 2)
    eye = torch.eye(hidden)
    o = torch.zeros(hidden, 2 * e)
    o[: 2 * e] = torch.eye(2 * e)
    tensors = {"q": eye[: 2 * d], "k": eye[2 * d: 3 * d], "v": eye[3 * d: 3 * d + e], "o": o, "q.norm": torch.ones(2 * d), "k.norm": torch.ones(d)}
    part, cache, step = mixer_harness(attention_spec(hidden, m), tensors, dtype, page_tokens=page, pages=200)
    gen = torch.Generator().manual_seed(d)
    for place in places_in(n, page):
        rows = torch.zeros(n, hidden)
        direction, others = torch.randn(d, generator=gen), torch.randn(n, d, generator=gen)
        direction[:2] = 0.0
        direction = torch.nn.functional.normalize(direction, dim=0)
        others -= (others @ direction)[:, None] * direction
        rows[:, 2 * d: 3 * d] = others
        rows[:, 3 * d: 3 * d + e] = 0.02 * torch.randn(n, e, generator=gen)
        rows[:, :d], rows[:, d: 2 * d] = direction, direction
        value = torch.randn(e, generator=gen)
        rows[place, 2 * d: 3 * d], rows[place, 3 * d: 3 * d + e] = 5 * direction, value
        rows = rows.to(dtype).float()
        want = plain.attention_mixer(rows.to(F), stored_as(tensors, dtype), m, 1e-5)
        assert float(want[n - 1, :e] @ value.to(F) / (value @ value)) > 0.9                # the test's own premise
        for name, cuts in {"whole": [n], "one decoded": [n - 1, 1], "uneven": _uneven(n)}.items():
            close(run_cuts(cache, step, rows, cuts)[n - 3:], want[n - 3:], dtype, f"key at {place}, {name}", slack=2)
    cache.check()


# ------------------------------------------------------------------ attention over a latent with latent queries
def latent_spec(hidden, m):
    rot = m["rot"]
    return PartSpec("latent_attention", dict(
        hidden=hidden, heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"], v_head_dim=m["vdim"], kv_rank=m["kv_rank"], q_rank=m["q_rank"],
        scale=m["scale"], norm_eps=1e-5, gate_kind="head", q_down="dq", q_down_norm="dq.norm", q="uq", down="dkv", down_norm="dkv.norm", up_k="uk",
        up_v="uv", gate="g", o="o", position=PartSpec("rotary_pairs", {"dim": m["rot_dim"], "theta": rot["base"], "rotated": rot["dims"],
                                                                       "ramp_scaling": rot.get("scaling")})))


def latent(heads, d, rot, e, rank, q_rank, scale, base, ramp=None):
    spec = {"base": base, "dims": rot}
    if ramp:
        spec["scaling"] = dict(zip(("factor", "original", "fast", "slow"), ramp))
    return {"heads": heads, "dim": d, "rot_dim": rot, "vdim": e, "kv_rank": rank, "q_rank": q_rank, "scale": scale, "rot": spec}


LATENT_SHAPES = [  # hidden, mixer, page; 17 and 20 heads take several groups of the decode kernel, rows above 256 the 32-bit kernel
    (40, latent(5, 10, 6, 14, 22, 18, 0.4, 3000.0, (5.0, 40, 9.0, 0.7)), 4), (64, latent(3, 32, 16, 48, 64, 40, 0.3, 40000.0, (3.0, 64, 16.0, 1.0)), 16),
    (96, latent(20, 24, 32, 16, 96, 72, 0.35, 700.0, (1.5, 500, 4.0, 1.5)), 8), (48, latent(1, 4, 2, 8, 4, 2, 1.0, 50.0, (2.0, 16, 2.0, 0.5)), 2),
    (64, latent(17, 16, 8, 8, 272, 24, 0.5, 700.0), 16), (38, latent(2, 12, 4, 6, 30, 50, 0.4, 100.0, (8.0, 30, 6.0, 0.3)), 4),
    (128, latent(4, 128, 64, 128, 192, 256, 0.07, 10000.0, (40.0, 4096, 32.0, 1.0)), 16)]


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("shape", LATENT_SHAPES)
def test_latent_attention_in_every_cut(dtype, shape):
    hidden, m, page = shape
    spec = latent_spec(hidden, m)
    tensors = random_tensors(build_part("mixer", spec, "").tensor_specs(), seed=m["kv_rank"], std=0.25)
    part, cache, step = mixer_harness(spec, tensors, dtype, page_tokens=page, pages=120)
    n = 90
    rows = torch.randn(n, hidden, generator=torch.Generator().manual_seed(6)).to(dtype).float()
    want = plain.latent_mixer(rows.to(F), stored_as(tensors, dtype), m, 1e-5)
    for name, cuts in cuts_of(n).items():
        close(run_cuts(cache, step, rows, cuts), want, dtype, name, slack=4)
    in_company(cache, step, rows, want, dtype, 4)


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("d, page", [(16, 4), (64, 16), (40, 8)])
def test_one_latent_among_hundreds(dtype, d, page):
    """As above: the last query's latent is the one key's latent, and every other latent is orthogonal to it. The rotated part
    of the queries is zero for one head; for the other it is what tells two equal latents at different positions apart."""
    rot, n = 8, 330
    hidden = 2 * d + rot + 8
    m = latent(2, d, rot, d, d, d, 9.0 / d, 300.0, (2.0, 40, 6.0, 1.0))
    eye = torch.eye(hidden)
    uq = torch.zeros(2 * (d + rot), d)
    uq[:d], uq[d + rot: 2 * d + rot] = torch.eye(d), torch.eye(d)
    uq[2 * d + rot:, :rot] = 0.5 * torch.eye(rot)
    o = torch.zeros(hidden, 2 * d)
    o[: min(hidden, 2 * d)] = torch.eye(2 * d)[: min(hidden, 2 * d)]
    g = torch.zeros(2, hidden)
    g[0, 2 * d + rot], g[1, 2 * d + rot] = 3.0, 0.5
    tensors = {"dq": eye[:d], "dq.norm": torch.ones(d), "uq": uq, "dkv": eye[d: 2 * d + rot], "dkv.norm": torch.ones(d),
               "uk": torch.eye(d).repeat(2, 1), "uv": torch.eye(d).repeat(2, 1), "g": g, "o": o}
    part, cache, step = mixer_harness(latent_spec(hidden, m), tensors, dtype, page_tokens=page, pages=200)
    gen = torch.Generator().manual_seed(d)
    for place in places_in(n, page):
        direction = torch.nn.functional.normalize(torch.randn(d, generator=gen), dim=0)
        others = torch.randn(n, d, generator=gen)
        others -= (others @ direction)[:, None] * direction
        rows = torch.zeros(n, hidden)
        rows[:, :d], rows[:, d: 2 * d] = direction, others
        rows[:, 2 * d: 2 * d + rot] = 0.3 * torch.randn(n, rot, generator=gen)
        rows[:, 2 * d + rot] = 1.0
        rows[place, d: 2 * d] = 4 * direction
        rows = rows.to(dtype).float()
        want = plain.latent_mixer(rows.to(F), stored_as(tensors, dtype), m, 1e-5)
        gate = torch.sigmoid(torch.tensor(3.0, dtype=F))
        share = float(want[n - 1, :d] @ direction.to(F)) / (d ** 0.5 * float(gate))
        assert share > 0.9                          # the test's own premise
        for name, cuts in {"whole": [n], "one decoded": [n - 1, 1], "uneven": _uneven(n)}.items():
            close(run_cuts(cache, step, rows, cuts)[n - 3:], want[n - 3:], dtype, f"latent at {place}, {name}", slack=2)
    cache.check()


# ------------------------------------------------------------------ routing, experts, the dense feed-forward
def routed_spec(hidden, experts, top, ff, limit, groups=None, keep=None, shared=None):
    return PartSpec("routed_experts", dict(
        hidden=hidden, experts=experts, top=top, inter=ff, activation="clipped_swiglu", limit=limit, slope=1.702, score="softmax_all", groups=groups,
        keep_groups=keep, group_score="best", renormalize=True, weight_on="output", router="router", expert_gate="e{}.gate", expert_up="e{}.up",
        expert_down="e{}.down", shared_gate="shared.sg" if shared else None,
        shared=PartSpec("gated_mlp", dict(hidden=hidden, inter=shared[0], activation="clipped_swiglu", limit=shared[1], slope=1.702, gate="shared.gate",
                                          up="shared.up", down="shared.down")) if shared else None))


def router_of(experts, top, groups, keep):
    return {"experts": experts, "top": top, **({"groups": {"count": groups, "keep": keep}} if groups else {})}


def firm_rows(h, router, spec, gap=1e-4):
    """The tokens whose choice of groups and of experts no rounding turns over."""
    logits = h.to(F) @ router.to(F).T
    firm, groups = torch.ones(h.shape[0], dtype=torch.bool), spec.get("groups")
    allowed = logits
    if groups and groups["keep"] < groups["count"]:
        best = logits.view(h.shape[0], groups["count"], -1).amax(dim=2)
        ranked = best.sort(dim=1, descending=True).values
        firm &= ranked[:, groups["keep"] - 1] - ranked[:, groups["keep"]] > gap
        kept = torch.zeros_like(best, dtype=torch.bool).scatter_(1, best.topk(groups["keep"], dim=1).indices, True)
        allowed = logits.masked_fill(~kept.repeat_interleave(spec["experts"] // groups["count"], dim=1), float("-inf"))
    if spec["top"] < spec["experts"]:
        ranked = allowed.sort(dim=1, descending=True).values
        firm &= ~(ranked[:, spec["top"] - 1] - ranked[:, spec["top"]] <= gap)
    return firm


ROUTES = [(16, 5, 4, 2, 64), (12, 3, 3, 1, 40), (5, 1, None, None, 24), (2, 2, 1, 1, 16), (1, 1, None, None, 16), (64, 8, 8, 3, 128),
          (130, 6, 13, 4, 72), (48, 40, 2, 2, 32), (6, 2, 6, 2, 48)]       # experts, top, groups, keep, hidden


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("tokens", [5, 150])
@pytest.mark.parametrize("route", ROUTES)
def test_the_choice_of_experts_and_their_weights(dtype, tokens, route):
    experts, top, groups, keep, hidden = route
    spec = routed_spec(hidden, experts, top, 8, 1.0, groups, keep)
    tensors = random_tensors(build_part("feed_forward", spec, "").tensor_specs(), seed=experts, std=0.5)
    part = bound_part("feed_forward", spec, tensors, dtype)
    h = torch.randn(tokens, hidden, generator=torch.Generator().manual_seed(experts * 7 + top)).to(dtype)
    ids, scores, factor = part.route(h.cuda())
    router = router_of(experts, top, groups, keep)
    want_ids, want_w = plain.route(h.to(F), tensors["router"].to(F), router)
    firm = firm_rows(h, tensors["router"], router)
    assert factor is None and firm.sum() >= tokens // 2
    got_ids, order = ids.cpu().long().sort(dim=1)
    ref_ids, ref_order = want_ids.sort(dim=1)
    assert torch.equal(got_ids[firm], ref_ids[firm])
    close(scores.cpu().gather(1, order)[firm], want_w.gather(1, ref_order)[firm], torch.float32, "weights", slack=30)
    close(scores.sum(dim=1), torch.ones(tokens, dtype=F), torch.float32, "the weights' sum")
    if groups:
        size = experts // groups
        assert all(len({int(e) // size for e in row}) <= keep for row in ids.cpu())


def test_a_groups_score_is_its_best_experts_alone():
    """Group 1 has the best expert and nothing else, group 0 two good ones: only group 1 takes part. Logits of hundreds stay
    finite; equal logits go to the lower index."""
    hidden, experts, top = 16, 6, 2
    router = torch.zeros(experts, hidden)
    router[:, 0] = torch.tensor([4.0, 4.0, 3.0, 5.0, -1.0, -2.0])
    router[:, 1] = torch.tensor([300.0, 299.0, -300.0, 298.0, 0.0, 100.0])
    spec = routed_spec(hidden, experts, top, 8, 1.0, 2, 1)
    part = bound_part("feed_forward", spec, dict(random_tensors(build_part("feed_forward", spec, "").tensor_specs(), 1), router=router), torch.float32)
    h = torch.zeros(3, hidden)
    h[0, 0], h[1, 1] = 1.0, 1.0
    ids, scores, _ = part.route(h.cuda())
    assert ids.cpu().tolist() == [[3, 4], [0, 1], [0, 1]]
    close(scores[0], torch.softmax(torch.tensor([5.0, -1.0], dtype=F), 0), torch.float32, "weights within the group")
    close(scores[1], torch.softmax(torch.tensor([300.0, 299.0], dtype=F), 0), torch.float32, "large logits")
    close(scores[2], torch.full((2,), 0.5, dtype=F), torch.float32, "equal logits")


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("tokens", [3, 40, 300])
@pytest.mark.parametrize("shape", [(64, 8, 3, 64, 1.5, 4, 2, (128, 0.7)), (40, 6, 2, 40, 0.5, 2, 1, (24, 1.5)), (76, 5, 1, 22, 2.0, None, None, None),
                                   (32, 2, 2, 8, 1.0, None, None, (64, 100.0)), (128, 12, 3, 128, 0.8, 3, 2, None),
                                   (48, 1, 1, 24, 100.0, None, None, (40, 0.9))])
def test_routed_experts_with_a_shared_expert(dtype, tokens, shape):
    """Few pairs and many, in both precisions: every form of the products, and the shared expert times its own gate, with a
    limit of its own."""
    hidden, experts, top, ff, limit, groups, keep, shared = shape
    spec = routed_spec(hidden, experts, top, ff, limit, groups, keep, shared)
    tensors = random_tensors(build_part("feed_forward", spec, "").tensor_specs(), seed=hidden + experts, std=0.35)
    part = bound_part("feed_forward", spec, tensors, dtype)
    h = torch.randn(tokens, hidden, generator=torch.Generator().manual_seed(tokens)).to(dtype)
    router = router_of(experts, top, groups, keep)
    mlp = {"router": router, "expert": {"limit": limit}, "shared": {"limit": shared[1]} if shared else None}
    stored = stored_as(tensors, dtype)
    want = plain.routed_feed_forward(h.to(F), stored, mlp)
    if shared:              # the test's own premise: the shared expert and its gate matter
        without = plain.routed_feed_forward(h.to(F), stored, dict(mlp, shared=None))
        assert (want - without).abs().max() > 0.05 * want.abs().max()
    got = part.forward(h.cuda()).float().cpu().to(F)
    wrong = ((got - want).abs().max(dim=1).values > 3 * tolerance(want.float(), dtype)) & firm_rows(h, tensors["router"], router)
    assert not bool(wrong.any()), f"{int(wrong.sum())} rows of {tokens} differ"


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("hidden, inter", [(48, 64), (64, 24), (128, 320), (256, 1024), (50, 7)])
def test_a_dense_feed_forward_with_a_clipped_gate(dtype, hidden, inter):
    """Up to 16 tokens and more than 128 have the gate in the product's epilogue where the width allows it (few-token kernel,
    single blocks, pairs of blocks), the steps between a kernel of their own; all of one arithmetic."""
    limit = 0.9
    spec = PartSpec("gated_mlp", dict(hidden=hidden, inter=inter, activation="clipped_swiglu", limit=limit, slope=1.702, gate="gate", up="up",
                                      down="down"))
    tensors = random_tensors(build_part("feed_forward", spec, "").tensor_specs(), seed=inter, std=2.0 / hidden ** 0.5)
    part = bound_part("feed_forward", spec, tensors, dtype)
    t = stored_as(tensors, dtype)
    for tokens in (1, 3, 16, 17, 128, 129, 300, 512, 700):
        h = torch.randn(tokens, hidden, generator=torch.Generator().manual_seed(tokens)).to(dtype)
        g, u = h.to(F) @ t["gate"].T, h.to(F) @ t["up"].T
        if tokens > 100:        # the test's own premise: each of the three cuts happens
            assert bool((g > limit).any()) and bool((u > limit).any()) and bool((u < -limit).any())
        close(part.forward(h.cuda()), plain.clipped_gate(h.to(F), t["gate"], t["up"], t["down"], limit), dtype, f"{tokens} tokens", slack=2)
    assert ops.gemm_status() == 0


# ------------------------------------------------------------------ whole models
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """name -> {"float32": (folder, raw config, weights), "bfloat16": the same model with firm routers}.

    Rounding to bfloat16 turns over a choice of experts wherever two logits lie that close; the token's row then moves by
    much of its size, and so do the rows of the tokens that look back at it. So the bfloat16 runs of whole models use routers
    whose choice rests on one channel that every token has alike: the embedding has a constant there, no sub-layer writes to
    it, and the mixes only scale it (the other channels still move the weights). Choices that depend on the token are
    compared in the 32-bit runs of whole models and, in both precisions, in the tests of the layer alone."""
    from safetensors.torch import load_file, save_file

    out = {}
    for name, raw in CONFIGS.items():
        folder = tmp_path_factory.mktemp(f"mimitar-{name}")
        # seeded by the name, so that a new configuration does not change the others' weights
        lb.write_model_folder(lb.MimitarConfig.from_hf_dict(raw), folder, seed=sum(map(ord, name)), **INIT[name])
        weights = load_file(str(folder / "model.safetensors"))
        firm_folder = tmp_path_factory.mktemp(f"mimitar-{name}-firm")
        firm = {k: v.clone() for k, v in weights.items()}
        firm["embed"][:, 0] = 0.6
        for key, value in weights.items():
            if key.endswith((".mix.o", ".down")):
                firm[key][0] = 0.0
            if key.endswith((".norm2", ".hc2.in")):
                firm[key] = value.abs() if key.endswith("in") else torch.where(torch.arange(value.numel()) == 0, torch.zeros_like(value), value)
            if key.endswith(".mlp.router"):
                order = torch.randperm(value.shape[0], generator=torch.Generator().manual_seed(value.shape[0]))
                firm[key] = (0.1 * value.float()).to(value.dtype)
                firm[key][:, 0] = 0.5 * (order - value.shape[0] / 2).to(value.dtype)
        save_file(firm, str(firm_folder / "model.safetensors"))
        (firm_folder / "config.json").write_text((folder / "config.json").read_text())
        raw_read = json.loads((folder / "config.json").read_text())
        out[name] = {"float32": (folder, raw_read, weights), "bfloat16": (firm_folder, raw_read, firm)}
    return out


LENGTHS = [1, 9, 70, 130, 33, 200]
_expected = {}
_moved = {}


def requests_for(name):
    return {f"r{i}": random_prompt(CONFIGS[name]["vocab"], n, seed=5 * len(name) + i) for i, n in enumerate(LENGTHS)}


def expected(folders, name, dtype_name):
    if (name, dtype_name) not in _expected:
        _, raw, weights = folders[name][dtype_name]
        _expected[name, dtype_name] = {rid: plain.forward(raw, weights, tokens)[0] for rid, tokens in requests_for(name).items()}
    return _expected[name, dtype_name]


def moved_by_rounding(folders, name):
    """Per request: how far rounding what a bfloat16 run stores moves each row of the plain model's logits."""
    if name not in _moved:
        _, raw, weights = folders[name]["bfloat16"]
        _moved[name] = {rid: plain.forward(raw, weights, tokens, plain.through_bfloat16)[0] - expected(folders, name, "bfloat16")[rid]
                        for rid, tokens in requests_for(name).items()}
    return _moved[name]


@pytest.mark.parametrize("dtype_name", list(DTYPES))
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("cut", list(CUTS))
def test_every_cut_matches_the_plain_implementation(folders, tmp_path, name, dtype_name, cut):
    folder = folders[name][dtype_name][0]
    steps = CUTS[cut](requests_for(name))
    if cut == "mixed":      # so few pages and slots that a request which ends hands both to the next one
        assert max_live_tokens(steps) < sum(-(-n // 64) * 64 for n in LENGTHS)
        assert max(len(s["entries"]) for s in steps) == 4
    rows = run_trace(folder, dtype_name, steps, tmp_path, block_tokens=PAGES[name], max_requests=4)
    compare(rows, expected(folders, name, dtype_name), DTYPES[dtype_name],
            moved_by_rounding(folders, name) if dtype_name == "bfloat16" else None)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_the_sum_of_the_streams_after_every_layer(folders, name):
    folder, raw, weights = folders[name]["float32"]
    tokens = random_prompt(raw["vocab"], 19, seed=2)
    _, after = plain.forward(raw, weights, tokens)
    model = lb.load_model(folder, dtype="float32")
    cache = lb.PagedKVCache(model, 32, block_tokens=PAGES[name], max_requests=2)
    builder = BatchBuilder(cache, model.device, model.tile_sizes())
    seq = cache.open("s")
    cache.grow(seq, len(tokens))
    taps = []

    def observe(index, x, delta):      # with what has not joined the streams yet
        assert x.dtype == torch.float32 and x.shape[1:] == (raw["streams"], raw["width"])
        taps.append(plain.write_streams(x.cpu().to(F), delta.mix.cpu().to(F), delta.gain.cpu().to(F), delta.value.cpu().to(F)).sum(dim=1))

    model.forward(builder.build([StepEntry(seq, tokens, [0])]), cache, observe=observe)
    assert len(taps) == after.shape[0]
    for run, (got, want) in enumerate(zip(taps, after)):
        close(got, want, torch.float32, f"layer {run}", slack=2)


@pytest.mark.parametrize("dtype_name", list(DTYPES))
@pytest.mark.parametrize("name", ["odd_sizes", "wide_heads"])
def test_long_decoding_on_few_pages(folders, tmp_path, name, dtype_name):
    """Seven tokens of prompt, then 180 decoded one by one, with just the pages and the one slot that they need."""
    folder, raw, weights = folders[name][dtype_name]
    tokens = random_prompt(raw["vocab"], 187, seed=9)
    want = plain.forward(raw, weights, tokens)[0]
    moved = {"long": plain.forward(raw, weights, tokens, plain.through_bfloat16)[0] - want} if dtype_name == "bfloat16" else None
    decoded = run_trace(folder, dtype_name, tail_decoded({"long": tokens}, tail=180), tmp_path / "decoded", max_tokens=192,
                        block_tokens=PAGES[name], max_requests=1)
    compare(decoded, {"long": want}, DTYPES[dtype_name], moved)


def test_32bit_logits_have_the_same_bits_in_every_cut(tmp_path):
    """Every sum of the 32-bit path runs in an order of its own, the shift's state included (not the experts', whose products
    have one form for few pairs and one for many)."""
    raw = config(90, 56, 2, [latent_layer(3, 12, 8, 16, 24, 20, 900.0, ramp=(4.0, 30, 6.0, 0.5), mlp=dense_mlp(72, 1.0)),
                             capped_layer(4, 2, 16, 24, 5000.0, 8, bands=(2.0, 1.0, 4.0, 50), softcap=6.0, mlp=dense_mlp(40, 1.5))], mult=0.8)
    folder = lb.write_model_folder(lb.MimitarConfig.from_hf_dict(raw), tmp_path / "model", seed=12, std=0.15, norm_std=0.3)
    requests = {f"r{n}": random_prompt(90, n, seed=n) for n in (33, 70, 130)}
    runs = [run_trace(folder, "float32", cut(requests), tmp_path / name, block_tokens=8, max_requests=4)
            for name, cut in {"portions": portions, "tail": tail_decoded, "mixed": mixed}.items()]
    for other in runs[1:]:
        for rid, rows in runs[0].items():
            for p, row in rows.items():
                assert np.array_equal(row, other[rid][p]), (rid, p)


@pytest.mark.parametrize("dtype_name", list(DTYPES))
@pytest.mark.parametrize("name", ["wide_heads", "many_streams"])
def test_replayed_graphs_give_the_rows_of_plain_launches(folders, tmp_path, name, dtype_name):
    folder = folders[name][dtype_name][0]
    steps = mixed({k: v for k, v in list(requests_for(name).items())[:4]})
    eager = run_trace(folder, dtype_name, steps, tmp_path / "a", block_tokens=16, max_requests=4)
    graphs = run_trace(folder, dtype_name, steps, tmp_path / "b", block_tokens=16, max_requests=4, cuda_graphs=True)
    for rid, rows in eager.items():
        for p, row in rows.items():
            other = graphs[rid][p]
            assert np.abs(row - other).max() <= (0.06 if dtype_name == "bfloat16" else 1e-3) * np.abs(row).max(), (rid, p)


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["odd_sizes", "wide_heads", "smallest"])
def test_greedy_generation_through_the_engine(folders, name, graphs):
    folder, raw, weights = folders[name]["float32"]
    model = lb.load_model(folder, dtype="float32")
    prompts = [random_prompt(raw["vocab"], n, seed=n) for n in (3, 21, 40, 8, 1)]
    got = lb.generate(model, prompts, max_new_tokens=12, block_tokens=PAGES[name], cuda_graphs=graphs,
                      config=lb.EngineConfig(max_batch=3, prefill_chunk=16, prefill_budget=16))
    for prompt, tokens in zip(prompts, got):
        assert len(tokens) == 12
        sequence = list(prompt)
        for token in tokens:
            logits = plain.forward(raw, weights, sequence)[0][-1]
            top = torch.topk(logits, 2).values
            if top[0] - top[1] > 1e-3 * logits.abs().max():     # a near tie may fall either way
                assert token == int(logits.argmax()), f"position {len(sequence)}"
            sequence.append(token)


def test_command_line_and_the_replay_program(folders, tmp_path):
    import subprocess
    import sys

    from conftest import ROOT

    folder, raw, weights = folders["odd_sizes"]["float32"]
    out = subprocess.run([sys.executable, "-m", "layover_b200", "--preset", "mimitar-tiny", "--random-weights", "--dtype", "bf16",
                          "--prompt-lens", "9,40", "--max-new-tokens", "4", "--num-blocks", "16", "--cuda-graphs"],
                         capture_output=True, text=True, cwd=ROOT, check=True)
    assert [len(g) for g in json.loads(out.stdout.strip().splitlines()[-1])["generated"]] == [4, 4]
    # the replay program as a program, on a folder whose config.json leaves the queries' rank to the stored tensors and
    # whose tensors include norms and connections that a layer without a feed-forward does not use
    from safetensors.torch import save_file

    stripped = json.loads((folder / "config.json").read_text())
    for entry in stripped["layers"]:
        entry["mixer"].pop("q_rank", None)
    other = tmp_path / "model"
    other.mkdir()
    (other / "config.json").write_text(json.dumps(stripped))
    unused = {"l3.norm2": torch.zeros(raw["width"]), **{f"l3.hc2.{k}": torch.zeros((3, 3) if k == "mix" else 3) for k in ("in", "out", "mix")}}
    save_file({**weights, **unused}, str(other / "model.safetensors"))
    requests = {f"q{i}": random_prompt(raw["vocab"], n, seed=60 + i) for i, n in enumerate([12, 30, 7, 19, 25])}
    steps = mixed(requests, live_limit=4)
    lines = "".join(json.dumps(s) + "\n" for s in steps)
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(other), "--dtype", "float32", "--out", str(tmp_path / "out"),
                          "--max-tokens", str(max_live_tokens(steps)), "--block-tokens", "4"],
                         input=lines, capture_output=True, text=True, cwd=ROOT, check=True)
    assert [l for l in run.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    compare(collect(steps, tmp_path / "out"), {rid: plain.forward(raw, weights, tokens)[0] for rid, tokens in requests.items()},
            torch.float32)
