"""A plain, slow Mimitar in float64 torch on the CPU: the oracle of the Mimitar tests.

One function per mechanism, written from the design's equations and sharing nothing with the package: every sequence
is taken alone and whole, with no cache, no pages and no batching. `forward` returns the logits of every position and
the sum of the residual streams after every layer run.

Notation: n tokens, W the model width, S residual streams, H query heads, G key/value heads, d the query/key size of a
head, e its value size, r a latent's size, E experts.
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


def rms_norm(x: torch.Tensor, weight, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def sub(tensors: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v.to(F) for k, v in tensors.items() if k.startswith(prefix)}


# ----------------------------------------------------------------------------- residual streams
def read_streams(streams: torch.Tensor, weights: torch.Tensor) -> torch.Tensor:
    """streams [n, S, W], weights [S] -> [n, W]: what a sub-layer is given."""
    return torch.einsum("nsw,s->nw", streams, weights)


def write_streams(streams: torch.Tensor, mix: torch.Tensor, gain: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """stream t <- sum over s of mix[s, t] stream s, + gain[t] y."""
    return torch.einsum("nsw,st->ntw", streams, mix) + gain[None, :, None] * y[:, None, :]


def shift(h: torch.Tensor, mu: torch.Tensor) -> torch.Tensor:
    """h [n, W]: every row moves towards the one before it (zeros before the first) by the share mu of each channel."""
    before = torch.cat((torch.zeros_like(h[:1]), h[:-1]))
    return h + (before - h) * mu


# ----------------------------------------------------------------------------- rotations
def banded_frequencies(rot: dict) -> torch.Tensor:
    """[dims / 2]: base^(-2 i / dims), rescaled by wavelength bands where the rotation has `scaling` {factor, low, high,
    original}: long waves slowed by the factor, short ones kept, a blend between."""
    scaling, out = rot.get("scaling"), []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if scaling:
            wave, original = 2 * math.pi / f, scaling["original"]
            if wave > original / scaling["low"]:
                f = f / scaling["factor"]
            elif wave >= original / scaling["high"]:
                s = (original / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=F)


def ramped_frequencies(rot: dict) -> tuple[torch.Tensor, float]:
    """(frequencies [dims / 2], the factor on cos and sin) with `scaling` {factor, original, fast, slow}: from the channel
    that turns `fast` times within `original` positions to the one that turns `slow` times, a ramp from the frequency
    itself to the frequency over `factor`; both cos and sin times 1 + 0.1 ln factor."""
    dims, base, scaling = rot["dims"], rot["base"], rot.get("scaling")
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(plain, dtype=F), 1.0

    def channel(turns):
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(channel(scaling["fast"])), 0), min(math.ceil(channel(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1 - ramp))
    return torch.tensor(out, dtype=F), 0.1 * math.log(scaling["factor"]) + 1.0


def turn_halves(x: torch.Tensor, freq: torch.Tensor) -> torch.Tensor:
    """x [n, heads, d], row p at position p: channel i turns with channel i + dims/2 (dims = 2 * freq's length)."""
    half = freq.numel()
    a = torch.arange(x.shape[0], dtype=F)[:, None, None] * freq
    u, v, rest = x[..., :half], x[..., half: 2 * half], x[..., 2 * half:]
    return torch.cat((u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin(), rest), dim=-1)


def turn_pairs(x: torch.Tensor, freq: torch.Tensor, factor: float) -> torch.Tensor:
    """x [n, heads, dims]: channel 2 i turns with channel 2 i + 1; cos and sin times `factor`."""
    a = torch.arange(x.shape[0], dtype=F)[:, None, None] * freq
    u, v = x[..., 0::2], x[..., 1::2]
    cos, sin = factor * a.cos(), factor * a.sin()
    return torch.stack((u * cos - v * sin, v * cos + u * sin), dim=-1).flatten(-2)


# ----------------------------------------------------------------------------- mixers
def causal_attention(q, k, v, scale: float, cap: float | None = None) -> torch.Tensor:
    """q [n, H, d], k [n, H, d], v [n, H, e] -> [n, H, e]; with a cap c a scaled score s becomes c tanh(s / c)."""
    n = q.shape[0]
    scores = torch.einsum("ihd,jhd->hij", q, k) * scale
    if cap:
        scores = cap * torch.tanh(scores / cap)
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return torch.einsum("hij,jhe->ihe", torch.softmax(scores.masked_fill((j > i)[None], float("-inf")), dim=-1), v)


def attention_mixer(h, t: dict, m: dict, eps: float, stored=exact) -> torch.Tensor:
    """Grouped-query attention: q and k normed over their whole rows, a partial banded rotation, capped scores."""
    n, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    freq = banded_frequencies(m["rot"])
    q = stored(turn_halves(rms_norm(h @ t["q"].T, t["q.norm"], eps).view(n, H, d), freq))
    k = stored(turn_halves(rms_norm(h @ t["k"].T, t["k.norm"], eps).view(n, G, d), freq))
    v = stored((h @ t["v"].T).view(n, G, e))
    out = causal_attention(q, k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1), m["scale"], m.get("softcap"))
    return stored(stored(out.reshape(n, H * e)) @ t["o"].T)


def latent_mixer(h, t: dict, m: dict, eps: float, stored=exact) -> torch.Tensor:
    """Attention whose queries and whose keys and values each come from a latent of the token; every head's output times
    a gate."""
    n, H, d, rot, e, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    freq, factor = ramped_frequencies(m["rot"])
    q = (stored(rms_norm(h @ t["dq"].T, t["dq.norm"], eps)) @ t["uq"].T).view(n, H, d + rot)
    down = h @ t["dkv"].T
    c = stored(rms_norm(down[:, :r], t["dkv.norm"], eps))
    k_rot = stored(turn_pairs(down[:, None, r:], freq, factor))
    q_rot = stored(turn_pairs(q[..., d:], freq, factor))
    k = torch.cat(((c @ t["uk"].T).view(n, H, d), k_rot.expand(n, H, rot)), dim=-1)
    v = (c @ t["uv"].T).view(n, H, e)
    out = causal_attention(torch.cat((stored(q[..., :d]), q_rot), dim=-1), k, v, m["scale"])
    out = stored(out) * torch.sigmoid(h @ t["g"].T)[:, :, None]
    return stored(stored(out.reshape(n, H * e)) @ t["o"].T)


MIXERS = {"attention": attention_mixer, "latent_attention": latent_mixer}


# ----------------------------------------------------------------------------- feed-forward
def clipped_gate(h, gate, up, down, limit: float, stored=exact) -> torch.Tensor:
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return stored(stored(g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.T)


def route(h, router: torch.Tensor, spec: dict):
    """(chosen experts [n, top], their weights [n, top]): softmax over all experts; only the groups with the largest
    single scores take part; the chosen scores over their sum."""
    scores = torch.softmax(h @ router.T, dim=-1)
    allowed, groups = scores.clone(), spec.get("groups")
    if groups:
        size = spec["experts"] // groups["count"]
        best = scores.view(-1, groups["count"], size).amax(dim=-1)
        kept = torch.zeros_like(best).scatter_(1, best.topk(groups["keep"], dim=-1).indices, 1.0)
        allowed = allowed.masked_fill(kept.repeat_interleave(size, dim=1) == 0, -1.0)
    chosen = allowed.topk(spec["top"], dim=-1).indices
    picked = scores.gather(1, chosen)
    return chosen, picked / (picked.sum(dim=-1, keepdim=True) + 1e-20)


def routed_feed_forward(h, t: dict, mlp: dict, stored=exact) -> torch.Tensor:
    chosen, weights = route(h, t["router"], mlp["router"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, place = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            y = clipped_gate(h[rows], t[f"e{e}.gate"], t[f"e{e}.up"], t[f"e{e}.down"], mlp["expert"]["limit"], stored)
            out.index_add_(0, rows, weights[rows, place][:, None] * y)
    if mlp.get("shared"):
        y = clipped_gate(h, t["shared.gate"], t["shared.up"], t["shared.down"], mlp["shared"]["limit"], stored)
        out = out + torch.sigmoid(h @ t["shared.sg"].T) * y
    return stored(out)


def feed_forward(h, t: dict, mlp: dict, stored=exact) -> torch.Tensor:
    if mlp["kind"] == "dense":
        return clipped_gate(h, t["gate"], t["up"], t["down"], mlp["limit"], stored)
    return routed_feed_forward(h, t, mlp, stored)


# ----------------------------------------------------------------------------- the model
def owner_of(config: dict, index: int) -> int:
    """The layer whose tensors layer `index` uses."""
    while config["layers"][index].get("weights_of") is not None:
        index = config["layers"][index]["weights_of"]
    return index


def forward(config: dict, tensors: dict, tokens: list[int], stored=exact):
    """(logits [n, vocab], the sum of the streams after every layer [layers, n, W]) of one whole sequence."""
    eps, m = config["norm"]["eps"], config["residual_mult"]
    embedded = tensors["embed"].to(F)[torch.tensor(tokens)]
    streams = embedded[:, None, :].expand(-1, config["streams"], -1)
    after = []
    for index, layer in enumerate(config["layers"]):
        t = sub(tensors, f"l{owner_of(config, index)}.")
        h = shift(rms_norm(read_streams(streams, t["hc1.in"]), 1 + t["norm1"], eps), t["shift"])
        y = MIXERS[layer["type"]](stored(h), sub(t, "mix."), layer["mixer"], eps, stored)
        streams = write_streams(streams, t["hc1.mix"], m * t["hc1.out"], y)
        if layer.get("mlp"):
            h = rms_norm(read_streams(streams, t["hc2.in"]), 1 + t["norm2"], eps)
            y = feed_forward(stored(h), sub(t, "mlp."), layer["mlp"], stored)
            streams = write_streams(streams, t["hc2.mix"], m * t["hc2.out"], y)
        after.append(streams.sum(dim=1))
    h = stored(rms_norm(streams.sum(dim=1), 1 + tensors["final.norm"].to(F), eps))
    return (h @ tensors["head"].to(F).T) * config.get("logit_scale", 1.0), torch.stack(after)
