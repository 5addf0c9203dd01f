"""Fimilix on the GPU against the plain implementation: every mechanism alone, then whole models in every way a
request can be cut, batched and decoded, in 32-bit and in bfloat16."""

import json
import math

import numpy as np
import pytest
import torch

import layover_b200 as lb
import plain_fimilix as plain
from conftest import random_prompt, tolerance
from fimilix_configs import CONFIGS, INIT, PAGES
from layover_b200 import ops
from layover_b200.cache import CacheManager
from layover_b200.engine.batch import BatchBuilder, StepEntry
from layover_b200.models.runtime import make_runtime
from layover_b200.parts.base import PartSpec, build_part, walk_parts
from replay_helpers import collect, max_live_tokens, mixed, portions, run_trace, tail_decoded, whole

pytestmark = pytest.mark.gpu
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F = torch.float64


def close(got: torch.Tensor, want: torch.Tensor, dtype, what="", slack=1.0):
    bound = slack * tolerance(want.float(), dtype)
    worst = (got.detach().cpu().to(F) - want.to(F)).abs().max().item()
    assert worst <= bound, f"{what}: |diff| {worst:.3e} > {bound:.3e}"


def bound_part(family, spec, tensors, dtype):
    runtime = make_runtime(dtype, "cuda")
    part = build_part(family, spec, "")
    from layover_b200.csrc import build
    build.ensure_built(tuple(n for p in walk_parts(part) for n in p.kernel_libraries(dtype)) + runtime.kernel_libraries)
    kinds = {s.name: s.kind for s in part.tensor_specs()}
    part.bind({k: v.to(dtype if kinds.get(k, "matrix") == "matrix" else torch.float32).cuda().contiguous()
               for k, v in tensors.items()}, runtime)
    return part


def stored_as(tensors: dict, dtype) -> dict:
    """The values a run of `dtype` holds (everything passes through it once)."""
    return {k: v.to(dtype).to(F) for k, v in tensors.items()}


def random_tensors(specs, seed, std=0.3):
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for s in specs:
        noise = torch.randn(s.shape, generator=gen)
        out[s.name] = ((1.0 + 0.3 * noise) if s.init == "ones" else std * noise).to(torch.bfloat16).float()
    return out


def mixer_harness(spec: PartSpec, tensors: dict, dtype, page_tokens=4, pages=96, slots=3):
    """One mixer part alone with its own cache manager and batch builder."""
    part = bound_part("mixer", spec, tensors, dtype)
    cache = CacheManager([(0, part.cache_need(), None)], pages, page_tokens, dtype, "cuda", slots, ops.RECORD_WORDS)
    sizes = tuple(s for p in walk_parts(part) for s in p.tile_sizes(dtype))
    builder = BatchBuilder(cache, torch.device("cuda"), sizes)

    def step(entries: list[tuple]):   # [(sequence, rows of h)] -> the mixer's output rows, per entry
        made = [StepEntry(seq, [0] * rows.shape[0], []) for seq, rows in entries]
        for entry in made:
            cache.grow(entry.seq, entry.seq.num_tokens + len(entry.tokens))
        batch = builder.build(made)
        out = part.forward(torch.cat([rows for _, rows in entries]).to(dtype).cuda().contiguous(), batch, cache.view(0))
        for entry in made:
            cache.commit(entry.seq, entry.seq.num_tokens + len(entry.tokens))
        return torch.split(out.float().cpu(), [rows.shape[0] for _, rows in entries])
    return part, cache, step


_names = iter(range(1 << 30))


def run_cuts(cache, step, rows: torch.Tensor, cuts: list[int]) -> torch.Tensor:
    seq, at, out = cache.open(f"s{next(_names)}"), 0, []
    for count in cuts:
        out.append(step([(seq, rows[at:at + count])])[0])
        at += count
    assert at == rows.shape[0]
    cache.close(seq)
    return torch.cat(out)


def _uneven(n: int) -> list[int]:
    out, sizes, i = [], (3, 2, 17, 5, 2, 40, 1, 64, 2, 9), 0
    while sum(out) < n:
        out.append(min(sizes[i % len(sizes)], n - sum(out)))
        i += 1
    return out


def cuts_of(n: int) -> dict[str, list[int]]:
    return {"whole": [n], "token by token": [1] * n, "pairs": [2] * (n // 2) + [1] * (n % 2),
            "half then single tokens": [n // 2] + [1] * (n - n // 2), "uneven": _uneven(n)}


def in_company(cache, step, rows, want, dtype, slack):
    """Two unequal requests at a time, one decoding while the other's prompt goes in; slots and pages are used again."""
    n = rows.shape[0]
    for _ in range(2):
        a, b = cache.open("a"), cache.open("b")
        first = step([(a, rows[:40])])[0]
        second = step([(a, rows[40:41]), (b, rows[:33])])
        third = step([(b, rows[33:n]), (a, rows[41:42])])
        close(torch.cat((first, second[0], third[1])), want[:42], dtype, "a beside b", slack=slack)
        close(torch.cat((second[1], third[0])), want, dtype, "b beside a", slack=slack)
        cache.close(b); cache.close(a)
    cache.check()


# ------------------------------------------------------------------ attention with capped scores and a query temperature
def attention_spec(hidden, heads, kv, d, e, scale, cap, temp, out_scale=1.0):
    return PartSpec("attention", dict(hidden=hidden, q_heads=heads, kv_heads=kv, head_dim=d, v_head_dim=e, scale=scale, softcap=cap,
                                      query_temperature=temp, qk_norm_eps=1e-5, out_scale=out_scale, exact_weights=True,
                                      q="q", k="k", v="v", o="o", q_norm="q.norm", k_norm="k.norm"))


def attention_mixer(heads, kv, d, e, scale, cap, temp) -> dict:
    return {"heads": heads, "kv_heads": kv, "dim": d, "vdim": e, "scale": scale, "softcap": cap,
            "q_temp": {"coef": temp[0], "every": temp[1]} if temp else None}


ATTENTION_SHAPES = [  # hidden, heads, kv, d, e, scale, cap, temperature, out_scale, page
    (40, 6, 2, 12, 20, 0.8, 4.0, (0.6, 7), 0.7, 4), (64, 4, 2, 32, 64, 0.4, 6.0, (0.3, 40), 1.0, 16),
    (64, 2, 1, 128, 128, 0.1, 3.0, (0.5, 16), 0.45, 16), (32, 20, 1, 8, 16, 0.5, 10.0, (2.0, 1), -1.5, 2),
    (48, 3, 3, 16, 16, 0.6, None, (0.9, 11), 1.0, 8), (48, 9, 1, 48, 16, 0.3, 2.0, None, 1.3, 16),
    (56, 2, 2, 160, 96, 0.1, 5.0, (0.4, 30), 0.8, 8), (64, 2, 1, 256, 256, 0.05, 3.0, (0.4, 30), 0.8, 16)]


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("shape", ATTENTION_SHAPES)
def test_attention_in_every_cut(dtype, shape):
    hidden, heads, kv, d, e, scale, cap, temp, out_scale, page = shape
    spec = attention_spec(hidden, heads, kv, d, e, scale, cap, temp, out_scale)
    tensors = random_tensors(build_part("mixer", spec, "").tensor_specs(), seed=d + e)
    part, cache, step = mixer_harness(spec, tensors, dtype, page_tokens=page, pages=120)
    n = 90
    rows = (torch.randn(n, hidden, generator=torch.Generator().manual_seed(5)) * 1.5).to(dtype).float()
    want = out_scale * plain.attention_mixer(rows.to(F), stored_as(tensors, dtype), attention_mixer(heads, kv, d, e, scale, cap, temp), 1e-5)
    for name, cuts in cuts_of(n).items():
        close(run_cuts(cache, step, rows, cuts), want, dtype, name, slack=3)
    in_company(cache, step, rows, want, dtype, 3)


def identity_attention(d, e, hidden):
    """Tensors with which a row of h IS [q (2 heads) | k | v] and the output row is [head 0 | head 1]."""
    eye = torch.eye(hidden)
    o = torch.zeros(hidden, 2 * e)
    o[: 2 * e] = torch.eye(2 * e)
    return {"q": eye[: 2 * d], "k": eye[2 * d: 3 * d], "v": eye[3 * d: 3 * d + e], "o": o,
            "q.norm": torch.ones(d), "k.norm": torch.ones(d)}


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("d, e, page", [(16, 16, 4), (64, 32, 16), (128, 128, 16), (12, 20, 4)])
def test_one_key_among_hundreds_and_what_the_cap_leaves_of_it(dtype, d, e, page):
    """The last query looks for ONE key, at the first position, at page and tile borders, far back and next to it. Uncapped
    its score would take all the weight; with a cap c the weight is e^c / (e^c + the rest), which the test's own premise
    checks, for a cap that leaves most of it and one that leaves little."""
    hidden, n = 3 * d + e + 4, 330
    gen = torch.Generator().manual_seed(d)
    tensors = identity_attention(d, e, max(hidden, 2 * e))
    hidden = max(hidden, 2 * e)
    last = n - 1
    shares = {}
    for cap in (9.0, 3.0):
        scale = 8.0 / d ** 0.5              # the matching pair scores 8 sqrt(d): far above either cap
        spec = attention_spec(hidden, 2, 1, d, e, scale, cap, None)
        part, cache, step = mixer_harness(spec, tensors, dtype, page_tokens=page, pages=200)
        for place in (0, page - 1, page, 31, 64, 65, last // page * page, last // page * page - 1, last - 1, last):
            rows = torch.zeros(n, hidden)
            direction = torch.nn.functional.normalize(torch.randn(d, generator=gen), dim=0)
            others = torch.randn(n, d, generator=gen)
            others -= (others @ direction)[:, None] * direction       # nothing of it in the other keys
            rows[:, 2 * d: 3 * d] = others
            rows[:, 3 * d: 3 * d + e] = 0.02 * torch.randn(n, e, generator=gen)
            for h in range(2):
                rows[:, h * d: (h + 1) * d] = direction
            value = torch.randn(e, generator=gen)
            rows[place, 2 * d: 3 * d], rows[place, 3 * d: 3 * d + e] = 5 * direction, value
            rows = rows.to(dtype).float()
            want = plain.attention_mixer(rows.to(F), stored_as(tensors, dtype), attention_mixer(2, 1, d, e, scale, cap, None), 1e-5)
            share = float(want[last, :e] @ value.to(F) / (value @ value))
            expected_share = math.exp(cap) / (math.exp(cap) + n - 1)
            assert abs(share - expected_share) < 0.15 * expected_share + 0.02, (share, expected_share)       # the test's own premise
            shares[cap] = share
            for name, cuts in {"whole": [n], "one decoded": [n - 1, 1], "uneven": _uneven(n)}.items():
                close(run_cuts(cache, step, rows, cuts)[last - 2:], want[last - 2:], dtype, f"cap {cap}, key at {place}, {name}", slack=2)
        cache.check()
    assert shares[9.0] > 0.9 and shares[3.0] < 0.1


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
def test_scores_far_beyond_a_cap_and_far_below_it(dtype):
    """Scores of +-thousands against a cap of 2, and of thousandths against a cap of 1000 (where capping changes nothing
    that a float holds): finite, and the plain softmax's."""
    heads, kv, d, e, hidden = 2, 1, 16, 16, 40
    for scale, cap in ((500.0, 2.0), (0.3, 1000.0), (1e-4, 50.0)):
        spec = attention_spec(hidden, heads, kv, d, e, scale, cap, None)
        tensors = random_tensors(build_part("mixer", spec, "").tensor_specs(), seed=3)
        part, cache, step = mixer_harness(spec, tensors, dtype)
        rows = torch.randn(70, hidden, generator=torch.Generator().manual_seed(1)).to(dtype).float()
        want = plain.attention_mixer(rows.to(F), stored_as(tensors, dtype), attention_mixer(heads, kv, d, e, scale, cap, None), 1e-5)
        for cuts in ([70], [40] + [1] * 30):
            got = run_cuts(cache, step, rows, cuts)
            assert torch.isfinite(got).all()
            # scores that reach +-cap with a slope of `scale` at zero: rounding a key moves a score near zero by much of the cap
            close(got, want, dtype, f"scale {scale}, cap {cap}", slack=60 if scale > 1 else 3)


@pytest.mark.parametrize("every, coef", [(1, 0.7), (5, 2.0), (64, 0.25), (1000, 3.0)])
def test_the_query_temperature_steps_where_position_plus_one_is_a_multiple(every, coef):
    positions = sorted({max(0, every * m + shift) for m in (1, 2, 3, 17) for shift in (-2, -1, 0)} | {0, 1, 2_000_000})
    n, d = len(positions), 8
    proj = torch.zeros(n, 3 * d, device="cuda")
    proj[:, :d] = 1.0
    q = torch.empty(n, d, device="cuda")
    pool = torch.zeros(n, 1, 1, d, device="cuda")
    ops.heads_bias_rope_kv(proj, q, pool, pool.clone(), None, None, None, None, torch.arange(n, dtype=torch.int32, device="cuda"), None, 0,
                           None, 1, 1, d, d, 1, temperature=(coef, every),
                           positions=torch.tensor(positions, dtype=torch.int32, device="cuda"))
    want = torch.tensor([1.0 + coef * math.log((p + 1) // every + 1) for p in positions], dtype=F)
    close(q[:, 0], want, torch.float32, "temperature", slack=1)
    at = {p: float(q[i, 0]) for i, p in enumerate(positions)}
    assert at[2 * every - 2] < at[2 * every - 1] == at[2 * every] or every == 1      # floor((p + 1) / every): the step is at p = 2 every - 1


# ------------------------------------------------------------------ gated linear attention
LINEAR_NAMES = dict(q="q", k="k", v="v", gate="g", a1="a1", a2="a2", a_bias="a2.b", norm="norm", o="o")
LINEAR_SHAPES = [  # hidden, heads, dim, vdim, rank, tau; sizes that are no multiple of 4 take the kernels' scalar forms
    (40, 3, 6, 10, 2, 3.0), (38, 5, 14, 9, 3, 16.0), (64, 2, 64, 32, 16, 8.0), (32, 1, 4, 4, 1, 1.0), (48, 4, 32, 72, 8, 30.0),
    (64, 1, 128, 96, 24, 5.0), (72, 2, 20, 64, 5, 2.0), (64, 1, 160, 16, 12, 10.0), (64, 2, 256, 40, 8, 0.5)]


def linear_spec(hidden, heads, d, e, rank, tau, out_scale=1.0):
    return PartSpec("gated_linear_attention", dict(hidden=hidden, heads=heads, head_dim=d, v_head_dim=e, decay_rank=rank, tau=tau,
                                                   norm_eps=1e-5, out_scale=out_scale, **LINEAR_NAMES))


def opposed_cancellation(tensors: dict) -> dict:
    """A head's output is normed, so a row whose terms cancel (the first token's o is (q . k) v) is decided by rounding.
    With k = q the first tokens' sums are squares."""
    return dict(tensors, k=tensors["q"].clone())


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("shape", LINEAR_SHAPES)
def test_gated_linear_attention_in_every_cut(dtype, shape):
    hidden, heads, d, e, rank, tau = shape
    spec = linear_spec(hidden, heads, d, e, rank, tau, out_scale=0.6)
    tensors = opposed_cancellation(random_tensors(build_part("mixer", spec, "").tensor_specs(), seed=d + e))
    part, cache, step = mixer_harness(spec, tensors, dtype)
    n = 90
    rows = torch.randn(n, hidden, generator=torch.Generator().manual_seed(5)).to(dtype).float()
    want = 0.6 * plain.linear_mixer(rows.to(F), stored_as(tensors, dtype), {"heads": heads, "dim": d, "vdim": e, "tau": tau}, 1e-5)
    slack = 3 if dtype == torch.bfloat16 else 20
    for name, cuts in cuts_of(n).items():
        close(run_cuts(cache, step, rows, cuts), want, dtype, name, slack=slack)
    in_company(cache, step, rows, want, dtype, slack)


def test_the_linear_scan_gives_the_same_bits_in_every_cut():
    hidden, heads, d, e, rank, tau = LINEAR_SHAPES[2]
    spec = linear_spec(hidden, heads, d, e, rank, tau)
    tensors = random_tensors(build_part("mixer", spec, "").tensor_specs(), seed=1)
    part, cache, step = mixer_harness(spec, tensors, torch.float32)
    rows = torch.randn(90, hidden, generator=torch.Generator().manual_seed(5))
    results = [run_cuts(cache, step, rows, cuts) for cuts in cuts_of(90).values()]
    assert all(torch.equal(results[0], r) for r in results[1:])


@pytest.mark.parametrize("wide", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tau", [0.5, 1.0, 16.0])
def test_decays_of_gates_from_shut_to_open(wide, tau):
    z = torch.tensor([-200.0, -60.0, -20.0, -5.0, -1e-3, 0.0, 1e-3, 5.0, 20.0, 60.0, 200.0])
    tokens, channels = 19, 5
    a = torch.zeros(tokens, 4, device="cuda")
    a[:, 0] = torch.tensor([float(z[t % z.numel()]) for t in range(tokens)])
    w2 = torch.zeros(channels, 1)
    w2[:, 0] = torch.tensor([1.0, 0.5, 0.0, -1.0, 0.25])
    bias = torch.tensor([0.0, 1.0, -3.0, 0.0, 2.0])
    got = torch.empty(tokens, channels, device="cuda")
    ops.gate_decay(a[:, :1], w2.to(wide).cuda(), bias.cuda(), tau, got)
    logits = a[:, :1].cpu().to(F) @ w2.to(F).T + bias.to(F)
    want = torch.exp(torch.nn.functional.logsigmoid(logits) / tau)
    assert torch.isfinite(got).all() and bool((got >= 0).all()) and bool((got <= 1).all())
    close(got, want, torch.float32, "decay", slack=1)


def test_the_state_remembers_or_forgets_by_channel_and_the_newest_write_is_read():
    """Identity projections, one head. Token 5 writes a pair (a, b); the last of 306 tokens asks for a. With open gates (a
    large bias) b comes back in the same direction, with half-shut ones nothing of it does. And a token that asks for the
    key it brings itself sees its own value."""
    d, rank = 16, 2
    hidden = 3 * d + 8
    eye = torch.eye(hidden)
    gate = torch.zeros(d, hidden)
    gate[:, 3 * d] = 2.0                                   # the same gate for every token and channel
    o = torch.zeros(hidden, d)
    o[:d] = torch.eye(d)
    base = {"q": eye[:d], "k": eye[d: 2 * d], "v": eye[2 * d: 3 * d], "g": gate, "o": o, "a1": torch.zeros(rank, hidden),
            "a2": torch.zeros(d, rank), "norm": torch.ones(d)}
    gen = torch.Generator().manual_seed(3)
    a, b, c = (torch.nn.functional.normalize(torch.randn(d, generator=gen), dim=0) for _ in range(3))
    n = 306
    rows = torch.randn(n, hidden, generator=gen) * 0.01
    rows[:, 3 * d] = 1.0
    rows[5, d: 2 * d], rows[5, 2 * d: 3 * d] = 4 * a, 4 * b
    rows[200, :d], rows[200, d: 2 * d], rows[200, 2 * d: 3 * d] = 4 * c, 4 * c, 4 * a       # its own write
    rows[n - 1, :d], rows[n - 1, d: 3 * d] = 4 * a - 4 * float(a @ c) * c, 0.0
    for bias, remembered in ((12.0, True), (0.0, False)):
        tensors = dict(base, **{"a2.b": torch.full((d,), bias)})
        part, cache, step = mixer_harness(linear_spec(hidden, 1, d, d, rank, 4.0), tensors, torch.float32)
        want = plain.linear_mixer(rows.to(F), stored_as(tensors, torch.float32), {"heads": 1, "dim": d, "vdim": d, "tau": 4.0}, 1e-5)
        for cuts in ([n], [200] + [1] * (n - 200), [3, 2] + [1] * (n - 5)):
            got = run_cuts(cache, step, rows, cuts)
            close(got, want, torch.float32, f"bias {bias}", slack=8)
            along = torch.nn.functional.cosine_similarity(got[n - 1, :d].to(F), b.to(F), dim=0)
            assert (along > 0.9) == remembered, float(along)
            own = torch.nn.functional.cosine_similarity(got[200, :d].to(F), a.to(F), dim=0)
            assert own > 0.9, float(own)


# ------------------------------------------------------------------ two mixers, one sum
@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("hidden, left, right", [
    (40, (3, 1, 12, 10), (2, 6, 7, 3)),            # rows of heads of 34 + 14: no multiple of 8; a width of 40
    (64, (4, 2, 32, 16), (2, 64, 32, 16)), (38, (2, 2, 16, 16), (3, 5, 9, 2))])
def test_scaled_mixers_side_by_side_over_one_product(dtype, hidden, left, right):
    (heads, kv, d, e), (lh, ld, le, rank) = left, right
    spec = PartSpec("side_by_side", {"hidden": hidden, "combine": "sum", "mixers": [
        (attention_spec(hidden, heads, kv, d, e, 0.5, 4.0, (0.5, 9), out_scale=0.7), "left.", None),
        (linear_spec(hidden, lh, ld, le, rank, 6.0, out_scale=-1.4), "right.", None)]})
    tensors = random_tensors(build_part("mixer", spec, "").tensor_specs(), seed=hidden)
    tensors["right.k"] = tensors["right.q"].clone()
    part, cache, step = mixer_harness(spec, tensors, dtype)
    n = 75
    rows = torch.randn(n, hidden, generator=torch.Generator().manual_seed(2)).to(dtype).float()
    want = plain.parallel_mixer(rows.to(F), stored_as(tensors, dtype), {
        "left": attention_mixer(heads, kv, d, e, 0.5, 4.0, (0.5, 9)), "right": {"heads": lh, "dim": ld, "vdim": le, "tau": 6.0},
        "left_scale": 0.7, "right_scale": -1.4}, 1e-5)
    slack = 3 if dtype == torch.bfloat16 else 20
    for name, cuts in cuts_of(n).items():
        close(run_cuts(cache, step, rows, cuts), want, dtype, name, slack=slack)
    in_company(cache, step, rows, want, dtype, slack)


# ------------------------------------------------------------------ norm, routing and experts
@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("width", [39, 1024])
def test_a_layer_norm_with_a_factor_on_its_output(dtype, width):
    gen = torch.Generator().manual_seed(width)
    x = torch.randn(5, width, generator=gen) * 3 + 7
    a, b = ((torch.randn(5, width, generator=gen)).to(dtype) for _ in range(2))
    w, bias = 1 + 0.3 * torch.randn(width, generator=gen), torch.randn(width, generator=gen)
    part = bound_part("norm", PartSpec("layernorm", {"dim": width, "eps": 1e-5, "weight": "w", "bias": "b", "out_scale": 0.3}),
                      {"w": w, "b": bias}, dtype)
    rows = torch.tensor([4, 0, 2], dtype=torch.int32, device="cuda")
    total = x.to(F) + a.to(F) + b.to(F)
    want = 0.3 * plain.layer_norm(total, w.to(F), bias.to(F), 1e-5)
    close(part.forward(x.cuda(), (a.cuda(), b.cuda()), rows=rows), want[[4, 0, 2]], dtype, "picked rows")
    close(part.forward(x.cuda(), (a.cuda(), b.cuda())), want, dtype, "all rows")


ROUTES = [(16, 5, 64), (7, 3, 40), (5, 1, 24), (2, 2, 16), (1, 1, 16), (64, 8, 128), (130, 6, 72), (48, 40, 32)]       # experts, top, hidden


def routed_spec(hidden, experts, top, ff, limit):
    return PartSpec("routed_experts", dict(
        hidden=hidden, experts=experts, top=top, inter=ff, activation="clipped_swiglu", limit=limit, slope=1.702, score="softmax",
        weight_on="output", router="router", expert_gate="e{}.gate", expert_up="e{}.up", expert_down="e{}.down"))


def firm_rows(h, router, top, gap):
    """The tokens whose choice of experts no rounding turns over."""
    logits = (h.to(F) @ router.to(F).T).sort(dim=1, descending=True).values
    if top == logits.shape[1]:
        return torch.ones(h.shape[0], dtype=torch.bool)
    return logits[:, top - 1] - logits[:, top] > gap


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("tokens", [5, 150])
@pytest.mark.parametrize("route", ROUTES)
def test_the_choice_of_experts_and_their_weights(dtype, tokens, route):
    experts, top, hidden = route
    spec = routed_spec(hidden, experts, top, 8, 1.0)
    tensors = random_tensors(build_part("feed_forward", spec, "").tensor_specs(), seed=experts, std=0.5)
    part = bound_part("feed_forward", spec, tensors, dtype)
    h = torch.randn(tokens, hidden, generator=torch.Generator().manual_seed(experts * 7 + top)).to(dtype)
    ids, scores, factor = part.route(h.cuda())
    want_ids, want_w = plain.route(h.to(F), tensors["router"].to(F), top)
    assert factor is None
    firm = firm_rows(h, tensors["router"], top, 1e-4)
    assert firm.sum() >= tokens // 2
    got_ids, order = ids.cpu().long().sort(dim=1)
    ref_ids, ref_order = want_ids.sort(dim=1)
    assert torch.equal(got_ids[firm], ref_ids[firm])
    close(scores.cpu().gather(1, order)[firm], want_w.gather(1, ref_order)[firm], torch.float32, "weights", slack=30)
    close(scores.sum(dim=1), torch.ones(tokens, dtype=F), torch.float32, "the weights' sum")


def test_routing_by_logits_far_apart_and_far_from_zero():
    """Logits of hundreds: the softmax over the chosen ones stays finite and the second expert's weight is exp of the gap."""
    hidden, experts, top = 16, 6, 3
    router = torch.zeros(experts, hidden)
    router[:, 0] = torch.tensor([300.0, 298.0, -300.0, 299.0, 0.0, 100.0])
    part = bound_part("feed_forward", routed_spec(hidden, experts, top, 8, 1.0),
                      dict(random_tensors(build_part("feed_forward", routed_spec(hidden, experts, top, 8, 1.0), "").tensor_specs(), 1), router=router),
                      torch.float32)
    h = torch.zeros(3, hidden)
    h[:, 0] = torch.tensor([1.0, -1.0, 0.0])
    ids, scores, _ = part.route(h.cuda())
    assert ids.cpu().tolist() == [[0, 3, 1], [2, 4, 5], [0, 1, 2]]         # ties: the lower index
    close(scores[0], torch.softmax(torch.tensor([300.0, 299.0, 298.0], dtype=F), 0), torch.float32, "large logits")
    close(scores[2], torch.full((3,), 1 / 3, dtype=F), torch.float32, "equal logits")


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("tokens", [3, 40, 300])
@pytest.mark.parametrize("shape", [(64, 8, 3, 64, 1.5), (40, 6, 2, 40, 0.5), (76, 5, 1, 22, 2.0), (32, 2, 2, 8, 1.0), (128, 12, 3, 128, 0.8),
                                   (48, 1, 1, 24, 100.0), (96, 10, 4, 192, 3.0)])
def test_routed_experts_with_clipped_gates(dtype, tokens, shape):
    """Few pairs (the weight-streaming kernels, and sizes they cannot read 16 bytes at a time), many in 32-bit (tiled
    FFMA), many in bfloat16 (grouped tensor-core products with the clipped gate in their epilogue, or behind them where
    the width is no multiple of 64). Gate and up logits reach several limits on either side."""
    hidden, experts, top, ff, limit = shape
    spec = routed_spec(hidden, experts, top, ff, limit)
    tensors = random_tensors(build_part("feed_forward", spec, "").tensor_specs(), seed=hidden + experts, std=0.35)
    part = bound_part("feed_forward", spec, tensors, dtype)
    assert part.interleaved == (dtype == torch.bfloat16 and ff % 64 == 0)
    h = torch.randn(tokens, hidden, generator=torch.Generator().manual_seed(tokens)).to(dtype)
    got = part.forward(h.cuda())
    mlp = {"router": {"experts": experts, "top": top}, "expert": {"limit": limit}}
    stored = stored_as(tensors, dtype)
    if limit < 50:          # the test's own premise: each of the three cuts happens
        g, u = h.to(F) @ stored["e0.gate"].T, h.to(F) @ stored["e0.up"].T
        assert bool((g > limit).any()) and bool((g < -limit).any()) and bool((u > limit).any()) and bool((u < -limit).any())
    want = plain.routed_feed_forward(h.to(F), stored, mlp)
    firm = firm_rows(h, tensors["router"], top, 1e-4)
    bound = 3 * tolerance(want.float(), dtype)
    wrong = ((got.float().cpu().to(F) - want).abs().max(dim=1).values > bound) & firm
    assert not bool(wrong.any()), f"{int(wrong.sum())} rows of {tokens} differ"


@pytest.mark.parametrize("dtype", list(DTYPES.values()))
@pytest.mark.parametrize("inter", [64, 24, 7])
def test_a_dense_feed_forward_takes_the_clipped_gate_too(dtype, inter):
    hidden, limit = 48, 0.9
    spec = PartSpec("gated_mlp", dict(hidden=hidden, inter=inter, activation="clipped_swiglu", limit=limit, slope=1.702, gate="gate", up="up",
                                      down="down"))
    tensors = random_tensors(build_part("feed_forward", spec, "").tensor_specs(), seed=inter, std=0.35)
    part = bound_part("feed_forward", spec, tensors, dtype)
    for tokens in (3, 200):
        h = torch.randn(tokens, hidden, generator=torch.Generator().manual_seed(tokens)).to(dtype)
        t = stored_as(tensors, dtype)
        close(part.forward(h.cuda()), plain.clipped_expert(h.to(F), t["gate"], t["up"], t["down"], limit), dtype, f"{tokens} tokens", slack=2)


# ------------------------------------------------------------------ whole models
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """name -> {"float32": (folder, raw config, weights), "bfloat16": the same model, well conditioned}.

    Rounding to bfloat16 turns over a choice of experts wherever two logits lie that close, and the direction of a normed
    head whose terms cancel; the token's row then moves by much of its size, and so do the rows of the tokens that look
    back at it. Random weights have such close calls every few dozen tokens. So the bfloat16 runs of whole models use
    routers whose choice rests on one constant channel of the norm's output (the same experts for every token; the other
    channels still move the weights) and linear attention with k = q, whose first sums are squares. Choices that depend on
    the token are compared in the 32-bit runs of whole models and, in both precisions, in the tests of the layer alone."""
    from safetensors.torch import load_file, save_file

    out = {}
    for name, raw in CONFIGS.items():
        folder = tmp_path_factory.mktemp(f"fimilix-{name}")
        # seeded by the name, so that a new configuration does not change the others' weights
        lb.write_model_folder(lb.FimilixConfig.from_hf_dict(raw), folder, seed=sum(map(ord, name)), **INIT[name])
        weights = {k: v.clone() for k, v in load_file(str(folder / "model.safetensors")).items()}
        for key, value in weights.items():
            if key.endswith(".a2.b"):
                value += 2.0            # gates that are open more often than shut: a memory of dozens of tokens
        save_file(weights, str(folder / "model.safetensors"))
        firm_folder = tmp_path_factory.mktemp(f"fimilix-{name}-firm")
        firm = {k: v.clone() for k, v in weights.items()}
        for key, value in weights.items():
            layer = key.split(".")[0] + "."
            if key.endswith(".mlp.router"):
                firm[layer + "norm1"][0], firm[layer + "norm1.b"][0] = 0.0, 1.0
                order = torch.randperm(value.shape[0], generator=torch.Generator().manual_seed(value.shape[0]))
                firm[key] = (0.1 * value.float()).to(value.dtype)
                firm[key][:, 0] = 1.5 * (order - value.shape[0] / 2).to(value.dtype)
            if key.endswith("mix.right.k"):
                firm[key] = weights[key[:-1] + "q"].clone()
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


def compare(rows, want, dtype, moved=None):
    for rid, reference in want.items():
        assert sorted(rows[rid]) == list(range(reference.shape[0])), f"{rid}: rows missing"
        got = torch.from_numpy(np.stack([rows[rid][p] for p in range(reference.shape[0])])).to(F)
        if dtype == torch.bfloat16:
            # a row's root mean square error against 1/16 of the spread of the row's logits (a key that is lost or a lost
            # state changes a row by about its own spread), or three times what rounding the stored tensors does to the
            # plain model's row, whichever is larger
            spread = (reference - reference.mean(dim=1, keepdim=True)).pow(2).mean(dim=1).sqrt()
            bound = torch.maximum(spread / 16, 3 * moved[rid].pow(2).mean(dim=1).sqrt())
            worst = (got - reference).pow(2).mean(dim=1).sqrt()
        else:
            bound = torch.full((reference.shape[0],), 8 * tolerance(reference.float(), dtype), dtype=F)
            worst = (got - reference).abs().max(dim=1).values
        bad = torch.nonzero(worst > bound)
        # a fault of a mask, a cache or a state breaks every row from some position on; bfloat16 rounding that happens to
        # fall badly on a row does not, so a few stray rows are let through in bfloat16: 3 in 100, and none by far
        allowed = max(2, reference.shape[0] * 3 // 100) if dtype == torch.bfloat16 else 0
        assert bad.numel() <= allowed and bool((worst <= 6 * bound).all()), \
            f"{rid}: {bad.numel()} wrong positions of {reference.shape[0]}, the first {int(bad[0])}: {worst[bad[0]].item():.3e} > {bound[bad[0]].item():.3e}"


CUTS = {"whole": whole, "tail": lambda r: tail_decoded(r, tail=40), "portions": portions, "mixed": mixed}


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
def test_the_stream_after_every_run_of_a_layer(folders, name):
    folder, raw, weights = folders[name]["float32"]
    tokens = random_prompt(raw["vocab"], 19, seed=2)
    _, after = plain.forward(raw, weights, tokens)
    model = lb.load_model(folder, dtype="float32")
    cache = lb.PagedKVCache(model, 32, block_tokens=PAGES[name], max_requests=2)
    builder = BatchBuilder(cache, model.device, model.tile_sizes())
    seq = cache.open("s")
    cache.grow(seq, len(tokens))
    taps = []

    def observe(index, x, delta):
        assert x.dtype == torch.float32
        taps.append(x.clone().to(F) + sum(d.to(F) for d in delta if d is not None))      # with what has not joined it yet

    model.forward(builder.build([StepEntry(seq, tokens, [0])]), cache, observe=observe)
    assert len(taps) == after.shape[0]
    for run, (got, want) in enumerate(zip(taps, after)):
        close(got, want, torch.float32, f"run {run}", slack=2)


@pytest.mark.parametrize("dtype_name", list(DTYPES))
@pytest.mark.parametrize("name", ["odd_sizes", "wide_heads"])
def test_long_decoding_on_few_pages(folders, tmp_path, name, dtype_name):
    """Seven tokens of prompt, then 180 decoded one by one, with just the pages and the one slot that they need: the
    recurrent states of every pass are carried 180 times and the temperature steps over decoded tokens."""
    folder, raw, weights = folders[name][dtype_name]
    tokens = random_prompt(raw["vocab"], 187, seed=9)
    want = plain.forward(raw, weights, tokens)[0]
    moved = {"long": plain.forward(raw, weights, tokens, plain.through_bfloat16)[0] - want} if dtype_name == "bfloat16" else None
    decoded = run_trace(folder, dtype_name, tail_decoded({"long": tokens}, tail=180), tmp_path / "decoded", max_tokens=192,
                        block_tokens=PAGES[name], max_requests=1)
    compare(decoded, {"long": want}, DTYPES[dtype_name], moved)


@pytest.mark.parametrize("dtype_name", list(DTYPES))
def test_replayed_graphs_give_the_rows_of_plain_launches(folders, tmp_path, dtype_name):
    folder = folders["wide_heads"][dtype_name][0]
    steps = mixed({k: v for k, v in list(requests_for("wide_heads").items())[:4]})
    eager = run_trace(folder, dtype_name, steps, tmp_path / "a", block_tokens=16, max_requests=4)
    graphs = run_trace(folder, dtype_name, steps, tmp_path / "b", block_tokens=16, max_requests=4, cuda_graphs=True)
    for rid, rows in eager.items():
        for p, row in rows.items():
            other = graphs[rid][p]
            assert np.abs(row - other).max() <= (0.06 if dtype_name == "bfloat16" else 1e-3) * np.abs(row).max(), (rid, p)


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["odd_sizes", "wide_heads"])
def test_greedy_generation_through_the_engine(folders, name, graphs):
    folder, raw, weights = folders[name]["float32"]
    model = lb.load_model(folder, dtype="float32")
    prompts = [random_prompt(raw["vocab"], n, seed=n) for n in (3, 21, 40, 8, 1)]
    got = lb.generate(model, prompts, max_new_tokens=12, block_tokens=PAGES[name], cuda_graphs=graphs,
                      config=lb.EngineConfig(max_batch=3, prefill_chunk=16, prefill_budget=16))
    for prompt, tokens in zip(prompts, got):
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
    out = subprocess.run([sys.executable, "-m", "layover_b200", "--preset", "fimilix-tiny", "--random-weights", "--dtype", "bf16",
                          "--prompt-lens", "9,40", "--max-new-tokens", "4", "--num-blocks", "16", "--cuda-graphs"],
                         capture_output=True, text=True, cwd=ROOT, check=True)
    assert [len(g) for g in json.loads(out.stdout.strip().splitlines()[-1])["generated"]] == [4, 4]
    # the replay program as a program, on a folder whose config.json leaves the decay rank to the stored tensors:
    # five requests through four state slots, one step at a time
    stripped = json.loads((folder / "config.json").read_text())
    for entry in stripped["layers"]:
        entry["mixer"]["right"].pop("decay_rank")
    other = tmp_path / "model"
    other.mkdir()
    (other / "config.json").write_text(json.dumps(stripped))
    (other / "model.safetensors").write_bytes((folder / "model.safetensors").read_bytes())
    requests = {f"q{i}": random_prompt(raw["vocab"], n, seed=60 + i) for i, n in enumerate([12, 30, 7, 19, 25])}
    steps = mixed(requests, live_limit=4)
    lines = "".join(json.dumps(s) + "\n" for s in steps)
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(other), "--dtype", "float32", "--out", str(tmp_path / "out"),
                          "--max-tokens", str(max_live_tokens(steps)), "--block-tokens", "4"],
                         input=lines, capture_output=True, text=True, cwd=ROOT, check=True)
    assert [l for l in run.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    compare(collect(steps, tmp_path / "out"), {rid: plain.forward(raw, weights, tokens)[0] for rid, tokens in requests.items()},
            torch.float32)
