"""A plain, slow Fimilix in float64 torch on the CPU: the oracle of the Fimilix tests.

One function per mechanism, written from the design's equations and sharing nothing with the package:
every sequence is taken alone and whole, token by token where the design is a recurrence, with no cache,
no pages and no batching. `forward` returns the logits of every position and the residual stream after
every layer run.

Notation: n tokens, W the model width, H query heads, G key/value heads, d the query/key size of a head,
e its value size, E experts.
"""

from __future__ import annotations

import math

import torch

F = torch.float64


def exact(t: torch.Tensor) -> torch.Tensor:
    return t


def through_bfloat16(t: torch.Tensor) -> torch.Tensor:
    """What a tensor becomes when it is stored in bfloat16 (inputs and outputs of matrix products in a
    bfloat16 run); the difference to the exact run says how far such rounding can move a row of logits."""
    return t.to(torch.bfloat16).to(F)


def layer_norm(x: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor, eps: float) -> torch.Tensor:
    mean = x.mean(dim=-1, keepdim=True)
    variance = ((x - mean) ** 2).mean(dim=-1, keepdim=True)
    return (x - mean) / torch.sqrt(variance + eps) * weight + bias


def rms_norm(x: torch.Tensor, weight, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def sub(tensors: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v.to(F) for k, v in tensors.items() if k.startswith(prefix)}


# ----------------------------------------------------------------------------- attention
def query_temperature(n: int, q_temp: dict | None) -> torch.Tensor:
    """[n]: 1 + coef ln(floor((p + 1) / every) + 1) for p = 0 .. n - 1 (1 without a temperature)."""
    if not q_temp:
        return torch.ones(n, dtype=F)
    return torch.tensor([1.0 + q_temp["coef"] * math.log((p + 1) // q_temp["every"] + 1) for p in range(n)], dtype=F)


def capped_attention(q, k, v, scale: float, cap: float | None) -> torch.Tensor:
    """q [n, H, d], k [n, H, d], v [n, H, e] (already one key/value head per query head) -> [n, H, e]: causal softmax
    over cap * tanh(score / cap)."""
    n = q.shape[0]
    scores = torch.einsum("ihd,jhd->hij", q, k) * scale
    if cap:
        scores = cap * torch.tanh(scores / cap)
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    scores = scores.masked_fill((j > i)[None], float("-inf"))
    return torch.einsum("hij,jhe->ihe", torch.softmax(scores, dim=-1), v)


def attention_mixer(h, t: dict, m: dict, eps: float, stored=exact) -> torch.Tensor:
    """Grouped-query attention without rotation: a norm per q and k head, a query temperature, capped scores."""
    n, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ t["q"].T).view(n, H, d), t["q.norm"], eps)
    k = rms_norm((h @ t["k"].T).view(n, G, d), t["k.norm"], eps)
    v = (h @ t["v"].T).view(n, G, e)
    q = stored(q * query_temperature(n, m.get("q_temp"))[:, None, None])
    k, v = stored(k).repeat_interleave(H // G, dim=1), stored(v).repeat_interleave(H // G, dim=1)
    out = capped_attention(q, k, v, m["scale"], m.get("softcap"))
    return stored(stored(out.reshape(n, H * e)) @ t["o"].T)


# ----------------------------------------------------------------------------- gated linear attention
def channel_decay(h, t: dict, heads: int, dim: int, tau: float) -> torch.Tensor:
    """alpha [n, H, d] in (0, 1): sigmoid(A2 (A1 h) + b)^(1 / tau)."""
    z = (h @ t["a1"].T) @ t["a2"].T + t["a2.b"]
    return (torch.sigmoid(z) ** (1.0 / tau)).view(h.shape[0], heads, dim)


def decayed_scan(q, k, v, alpha) -> torch.Tensor:
    """q, k, alpha [n, H, d], v [n, H, e]: per head S <- diag(alpha_t) S + k_t v_t^T, then o_t = S^T q_t."""
    n, H, d = q.shape
    S = torch.zeros((H, d, v.shape[-1]), dtype=F)
    out = torch.zeros((n, H, v.shape[-1]), dtype=F)
    for i in range(n):
        S = alpha[i][:, :, None] * S + k[i][:, :, None] * v[i][:, None, :]
        out[i] = torch.einsum("hde,hd->he", S, q[i])
    return out


def linear_mixer(h, t: dict, m: dict, eps: float, stored=exact) -> torch.Tensor:
    n, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ t["q"].T).view(n, H, d) / math.sqrt(d)
    k = (h @ t["k"].T).view(n, H, d)
    v = (h @ t["v"].T).view(n, H, e)
    o = decayed_scan(q, k, v, channel_decay(h, t, H, d, m["tau"]))
    o = rms_norm(o, t["norm"], eps).reshape(n, H * e) * silu(h @ t["g"].T)
    return stored(stored(o) @ t["o"].T)


def parallel_mixer(h, t: dict, m: dict, eps: float, stored=exact) -> torch.Tensor:
    return (m["left_scale"] * attention_mixer(h, sub(t, "left."), m["left"], eps, stored)
            + m["right_scale"] * linear_mixer(h, sub(t, "right."), m["right"], eps, stored))


# ----------------------------------------------------------------------------- feed-forward
def clipped_expert(h, gate, up, down, limit: float, stored=exact) -> torch.Tensor:
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return stored(stored(g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.T)


def route(h, router: torch.Tensor, top: int):
    """(chosen experts [n, top], their weights [n, top]): the largest logits, softmax over the chosen ones."""
    values, chosen = (h @ router.T).topk(top, dim=-1)
    return chosen, torch.softmax(values, dim=-1)


def routed_feed_forward(h, t: dict, mlp: dict, stored=exact) -> torch.Tensor:
    chosen, weights = route(h, t["router"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, place = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            y = clipped_expert(h[rows], t[f"e{e}.gate"], t[f"e{e}.up"], t[f"e{e}.down"], mlp["expert"]["limit"], stored)
            out.index_add_(0, rows, weights[rows, place][:, None] * y)
    return stored(out)


# ----------------------------------------------------------------------------- the model
def layer_order(config: dict) -> list[int]:
    """The layers in the order they run: the loop's span `times` times in a row."""
    order = list(range(len(config["layers"])))
    loop = config.get("loop")
    if not loop:
        return order
    span = order[loop["start"]: loop["stop"]]
    return order[: loop["start"]] + span * loop["times"] + order[loop["stop"]:]


def forward(config: dict, tensors: dict, tokens: list[int], stored=exact):
    """(logits [n, vocab], the stream after every layer run [runs, n, W]) of one whole sequence."""
    eps = config["norm"]["eps"]
    x = tensors["embed"].to(F)[torch.tensor(tokens)]
    streams = []
    for index in layer_order(config):
        layer, t = config["layers"][index], sub(tensors, f"l{index}.")
        h = stored(layer_norm(x, t["norm1"], t["norm1.b"], eps))
        out = parallel_mixer(h, sub(t, "mix."), layer["mixer"], eps, stored)
        if layer.get("mlp"):
            out = out + routed_feed_forward(h, sub(t, "mlp."), layer["mlp"], stored)
        x = x + out
        streams.append(x.clone())
    h = stored(layer_norm(x, tensors["final.norm"].to(F), tensors["final.norm.b"].to(F), eps))
    return (h @ tensors["head"].to(F).T) * config.get("logit_scale", 1.0), torch.stack(streams)
