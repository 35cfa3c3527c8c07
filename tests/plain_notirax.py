"""The Notirax decoder written out slowly: whole sequences, no cache, torch on the CPU in float64.

One function per mechanism. It shares no code with ``infer_b200``: it reads the raw config.json dictionary and a
dictionary of checkpoint tensors by their names in the file. Everything the engine does for this design is compared
with this file.

The token table's rows plus a sinusoidal position vector (``sinusoid``) fill n equal residual streams x_1 .. x_n. A
sublayer f (mixer or feed-forward) reads one combination of the streams and writes into all of them (``link``):

    u = sum_s a_s x_s;   y = f(norm(u));   x_t <- sum_s M[s, t] x_s + b_t y      (all t from the old x)

and the logits are table . norm(sum_s x_s). The norm (``grouped_norm``) divides each of several equal parts of a row by
the part's own root mean square. Mixers: ``talking_attention`` (capped scores that the heads exchange through a matrix
before the softmax, keys of the query's own chunk only) and ``channel_delta_rule`` (a delta rule whose state fades by a
number per head, key channel and token). Feed-forward: ``routed_experts`` with sigmoid scores and groups.

``ROUNDING``: None computes exactly. Set to ``torch.bfloat16`` (see ``rounded``), activations are rounded where a
bfloat16 serving path stores them, which gives the size of the rounding noise such a path must have.
"""
from __future__ import annotations

import math
from typing import Dict, List, Mapping, Optional, Sequence

import torch

F = torch.float64
POSITION_BASE = 10000.0
UNIT_EPS = 1e-6
EXPERT_SLOPE = 1.702

ROUNDING = None


class rounded:
    """with rounded(torch.bfloat16): ... computes with activations rounded where a serving path stores them."""

    def __init__(self, dtype):
        self.dtype = dtype

    def __enter__(self):
        global ROUNDING
        self.old, ROUNDING = ROUNDING, self.dtype

    def __exit__(self, *exc):
        global ROUNDING
        ROUNDING = self.old


def _rnd(x: torch.Tensor) -> torch.Tensor:
    return x if ROUNDING is None else x.to(ROUNDING).to(x.dtype)


def linear(x: torch.Tensor, W: torch.Tensor, b: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = x @ W.to(F).T
    return y if b is None else y + b.to(F)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ----------------------------------------------------------------------------- the stream

def sinusoid(positions: torch.Tensor, width: int) -> torch.Tensor:
    """[T, width]: channels 2i and 2i + 1 hold sin and cos of position * POSITION_BASE^(-2i / width)."""
    c = torch.arange(width)
    freq = POSITION_BASE ** (-(c - c % 2).to(F) / width)
    a = positions.to(F)[:, None] * freq[None, :]
    return torch.where((c % 2 == 0)[None, :], torch.sin(a), torch.cos(a))


def grouped_norm(x: torch.Tensor, w: torch.Tensor, eps: float, groups: int) -> torch.Tensor:
    """Each of ``groups`` consecutive parts of a row over its own root mean square, then a weight per channel."""
    parts = x.reshape(*x.shape[:-1], groups, -1)
    parts = parts / torch.sqrt((parts * parts).mean(dim=-1, keepdim=True) + eps)
    return parts.reshape(x.shape) * w.to(F)


def read_streams(X: torch.Tensor, a: torch.Tensor) -> torch.Tensor:
    """X [T, n, width], a [n] -> [T, width]."""
    return torch.einsum("tsc,s->tc", X, a.to(F))


def write_streams(X: torch.Tensor, M: torch.Tensor, b: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """M is [from, to]."""
    return torch.einsum("tsc,sr->trc", X, M.to(F)) + b.to(F)[None, :, None] * y[:, None, :]


def link(X: torch.Tensor, W: Mapping[str, torch.Tensor], p: str, norm_w: torch.Tensor, eps: float, groups: int, sublayer) -> torch.Tensor:
    h = _rnd(grouped_norm(read_streams(X, W[p + "in"]), norm_w, eps, groups))
    return write_streams(X, W[p + "mix"], W[p + "out"], sublayer(h))


# ----------------------------------------------------------------------------- attention

def softcap(s: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return s if not cap else cap * torch.tanh(s / cap)


def visible(T: int, chunk: Optional[int]) -> torch.Tensor:
    """[T, T] bool: query i sees key j if j <= i and both lie in one chunk of ``chunk`` positions (None: any j <= i)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok if chunk is None else ok & (i // chunk == j // chunk)


def exchange_heads(s: torch.Tensor, talk: torch.Tensor) -> torch.Tensor:
    """s [heads, ...]: head h becomes sum over g of talk[h, g] s_g."""
    return torch.einsum("hg,g...->h...", talk.to(F), s)


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, cap: Optional[float], talk: Optional[torch.Tensor],
           seen: torch.Tensor) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]."""
    H, r = q.shape[1], q.shape[1] // k.shape[1]
    s = torch.stack([q[:, h] @ k[:, h // r].T * scale for h in range(H)])
    s = softcap(s, cap)
    if talk is not None:
        s = exchange_heads(s, talk)
    p = torch.softmax(s.masked_fill(~seen[None], -math.inf), dim=-1)
    return torch.stack([p[h] @ v[:, h // r] for h in range(H)], dim=1)


def talking_attention(h: torch.Tensor, W: Mapping[str, torch.Tensor], p: str, m: Mapping) -> torch.Tensor:
    H, G, d = int(m["heads"]), int(m.get("kv_heads") or m["heads"]), int(m["dim"])
    dv, T = int(m.get("vdim") or d), h.shape[0]
    q = _rnd(linear(h, W[p + "q"], W[p + "q.b"])).view(T, H, d)
    k = _rnd(linear(h, W[p + "k"], W[p + "k.b"])).view(T, G, d)
    v = _rnd(linear(h, W[p + "v"], W[p + "v.b"])).view(T, G, dv)
    mask = m.get("mask")
    o = attend(q, k, v, float(m["scale"]), m.get("softcap"), W[p + "talk"], visible(T, int(mask["size"]) if mask else None))
    return linear(_rnd(o).reshape(T, H * dv), W[p + "o"], W[p + "o.b"])


# ----------------------------------------------------------------------------- the delta rule

def causal_filter(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the sequence."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=F), u])
    return sum(padded[j:j + u.shape[0]] * w[:, j].to(F) for j in range(taps))


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + UNIT_EPS)


def channel_delta_scan(q, k, v, g, beta, S=None):
    """One head: q, k, g [T, d], v [T, dv], beta [T] -> (o [T, dv], final state [d, dv])."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=F) if S is None else S.clone()
    out = []
    for t in range(q.shape[0]):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + k[t][:, None] * u[None, :]
        out.append(S.T @ q[t])
    return torch.stack(out), S


def channel_decays(z: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor, heads: int) -> torch.Tensor:
    """z [T, heads * d] -> exp(-exp(a_log of the head) softplus(z + dt_bias)), [T, heads, d]."""
    s = torch.nn.functional.softplus(z + dt_bias.to(F)).view(z.shape[0], heads, -1)
    return torch.exp(-torch.exp(a_log.to(F))[None, :, None] * s)


def channel_delta_rule(h: torch.Tensor, W: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float) -> torch.Tensor:
    H, G, d = int(m["heads"]), int(m.get("kv_heads") or m["heads"]), int(m["dim"])
    dv, T, r = int(m.get("vdim") or d), h.shape[0], int(m["heads"]) // int(m.get("kv_heads") or m["heads"])
    f = (lambda u, n: causal_filter(u, W[p + n + ".conv"])) if m.get("conv") else (lambda u, n: u)
    q = silu(f(linear(h, W[p + "q"]), "q")).view(T, G, d)
    k = silu(f(linear(h, W[p + "k"]), "k")).view(T, G, d)
    v = silu(f(linear(h, W[p + "v"]), "v")).view(T, H, dv)
    q, k = unit(q) * d ** -0.5, unit(k)
    beta = torch.sigmoid(linear(h, W[p + "b"]))
    g = channel_decays(linear(_rnd(linear(h, W[p + "a1"])), W[p + "a2"]), W[p + "A_log"], W[p + "dt_bias"], H)
    o = torch.stack([channel_delta_scan(q[:, i // r], k[:, i // r], v[:, i], g[:, i], beta[:, i])[0] for i in range(H)], dim=1)
    o = o / torch.sqrt((o * o).mean(dim=-1, keepdim=True) + eps) * W[p + "norm"].to(F)
    gate = torch.sigmoid(linear(_rnd(linear(h, W[p + "g1"])), W[p + "g2"]))
    return linear(_rnd(o.reshape(T, H * dv) * gate), W[p + "o"])


# ----------------------------------------------------------------------------- feed-forward

def group_scores(s: torch.Tensor, groups: int) -> torch.Tensor:
    """s [T, E]: per group of neighbours the sum of its two largest scores (of its one, if it has one)."""
    per = s.shape[1] // groups
    return s.view(-1, groups, per).topk(min(2, per), dim=-1).values.sum(dim=-1)


def route(z: torch.Tensor, router: Mapping, gaps: Optional[List] = None):
    """Logits [T, E] -> (chosen [T, top], weights [T, top]). ``gaps`` collects, per token, the smallest distance
    between a score (of a group or an expert) that was chosen and one that was not."""
    E, top = z.shape[1], int(router["top"])
    groups = router.get("groups") or {"count": 1, "keep": 1}
    count, keep = int(groups["count"]), int(groups["keep"])
    s = torch.sigmoid(z)
    gs = group_scores(s, count)
    kept = gs.topk(keep, dim=-1).indices
    allowed = torch.zeros(z.shape[0], count, dtype=torch.bool).scatter_(1, kept, True).repeat_interleave(E // count, dim=1)
    masked = s.masked_fill(~allowed, -1.0)
    chosen = masked.topk(top, dim=-1).indices
    if gaps is not None:
        gap = torch.full((z.shape[0],), math.inf, dtype=F)
        if keep < count:
            o = gs.sort(dim=-1, descending=True).values
            gap = torch.minimum(gap, o[:, keep - 1] - o[:, keep])
        if top < keep * (E // count):
            o = masked.sort(dim=-1, descending=True).values
            gap = torch.minimum(gap, o[:, top - 1] - o[:, top])
        gaps.append(gap)
    return chosen, s.gather(1, chosen) * float(router.get("scale", 1.0))


def clipped_expert(x: torch.Tensor, W: Mapping[str, torch.Tensor], u: str, limit: float, weight=1.0) -> torch.Tensor:
    g = torch.clamp(_rnd(linear(x, W[u + "gate"])), max=limit)
    y = torch.clamp(_rnd(linear(x, W[u + "up"])), -limit, limit)
    return linear(_rnd(g * torch.sigmoid(EXPERT_SLOPE * g) * (y + 1.0) * weight), W[u + "down"])


def routed_experts(h: torch.Tensor, W: Mapping[str, torch.Tensor], p: str, f: Mapping, gaps: Optional[List] = None) -> torch.Tensor:
    chosen, weights = route(linear(h, W[p + "router"]), f["router"], gaps)
    out = torch.zeros_like(h)
    for e in range(int(f["router"]["experts"])):
        t, slot = torch.nonzero(chosen == e, as_tuple=True)
        if len(t):
            out[t] += clipped_expert(h[t], W, p + f"e{e}.", float(f["expert"]["limit"]), weights[t, slot][:, None])
    return out


# ----------------------------------------------------------------------------- the model

def forward(cfg: Mapping, W: Mapping[str, torch.Tensor], ids: Sequence[int], layer_outputs: Optional[List] = None,
            gaps: Optional[List] = None) -> torch.Tensor:
    """Logits [T, vocab] (float64) of one sequence; ``layer_outputs`` collects the sum of the streams after every layer,
    ``gaps`` every router's close calls (see ``route``)."""
    eps, groups, n = float(cfg["norm"]["eps"]), int(cfg["norm"].get("groups") or 1), int(cfg.get("streams") or 1)
    T = len(ids)
    x = W["embed"].to(F)[torch.tensor(list(ids), dtype=torch.long)] + sinusoid(torch.arange(T), int(cfg["width"]))
    X = x[:, None, :].repeat(1, n, 1)
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        if layer["type"] == "attention":
            mix = lambda h: talking_attention(h, W, p + "mix.", m)
        elif layer["type"] == "channel_delta":
            mix = lambda h: channel_delta_rule(h, W, p + "mix.", m, eps)
        else:
            raise ValueError(f"unknown layer type {layer['type']!r}")
        X = link(X, W, p + "hc1.", W[p + "norm1"], eps, groups, mix)
        if f is not None:
            X = link(X, W, p + "hc2.", W[p + "norm2"], eps, groups, lambda h: routed_experts(h, W, p + "mlp.", f, gaps))
        if layer_outputs is not None:
            layer_outputs.append(X.sum(dim=1))
    return linear(_rnd(grouped_norm(X.sum(dim=1), W["final.norm"], eps, groups)), W["embed"])


def greedy(cfg: Mapping, W: Mapping[str, torch.Tensor], prompt: Sequence[int], n_new: int) -> List[int]:
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(torch.argmax(forward(cfg, W, ids)[-1])))
    return ids[len(prompt):]
