"""The Bolelix decoder written out slowly: whole sequences, no cache, torch on the CPU in float64.

One function per mechanism. It shares no code with ``infer_b200``: it reads the raw config.json dictionary and a
dictionary of checkpoint tensors by their names in the file. Everything the engine does for this design is compared
with this file.

The residual stream x starts as table[token] * embedding.scale. A layer has one norm, whose rows both sublayers read:

    n = norm(x);    x <- x + ls1 * mixer(n) + ls2 * feed_forward(n)         (ls1, ls2: a stored factor per channel)

Mixers: ``state_space`` (layer type "mamba2": a filter over time in front of a matrix state per head that fades by one
number per head and token; a gate before a norm over groups), ``windowed_attention`` (type "attention": rotation of
channels i and i + dims / 2, unit-root-mean-square queries and keys, a window that keeps the first tokens, one gate per
head, keys and values that may be another layer's) and ``matrix_memory`` (type "mlstm": exponential input gates and
forget gates with a running maximum, a normaliser beside the state). Feed-forward: ``routed_experts``.

``ROUNDING``: None computes exactly. Set to ``torch.bfloat16`` (see ``rounded``), activations are rounded where a
bfloat16 serving path stores them, which gives the size of the rounding noise such a path must have.
"""
from __future__ import annotations

import math
from typing import Dict, List, Mapping, Optional, Sequence

import torch

F = torch.float64
DENOMINATOR_FLOOR = 1e-6       # added to the matrix memory's normaliser

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


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * w.to(F)


def linear(x: torch.Tensor, W: torch.Tensor) -> torch.Tensor:
    return x @ W.to(F).T


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    """ln(1 + e^z)."""
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    return -softplus(-z)


# ----------------------------------------------------------------------------- attention

def frequencies(dims: int, base: float, factor: float) -> torch.Tensor:
    """base^(-2i / dims) / factor for the dims / 2 channel pairs."""
    return base ** (-2.0 * torch.arange(dims // 2, dtype=F) / dims) / factor


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, rot: Mapping) -> torch.Tensor:
    """x [T, heads, dim]: channel i below dims / 2 turns together with channel i + dims / 2; channels from dims on pass."""
    dims = int(rot["dims"])
    scaling = rot.get("scaling")
    a = positions.to(F)[:, None] * frequencies(dims, float(rot["base"]), float(scaling["factor"]) if scaling else 1.0)[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def visible(T: int, window: Optional[int], keep_first: int) -> torch.Tensor:
    """[T, T] bool: query i sees key j if j <= i and (i - j < window or j < keep_first); no window: every j <= i."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    if window is not None:
        ok = ok & ((i - j < window) | (j < keep_first))
    return ok


def _rotated_unit(x: torch.Tensor, rot: Optional[Mapping], eps: float) -> torch.Tensor:
    """Rotation first, then every head over its own root mean square."""
    if rot:
        x = rotate_halves(x, torch.arange(x.shape[0]), rot)
    return rms(x, eps)


def windowed_attention(h, W: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float, shared: Optional[Dict[int, tuple]] = None,
                       index: int = 0) -> torch.Tensor:
    """``shared`` collects (keys, values) per layer index; a mixer with ``kv_from`` reads an earlier layer's there."""
    T = h.shape[0]
    H, G, d = int(m["heads"]), int(m.get("kv_heads") or m["heads"]), int(m["dim"])
    dv = int(m.get("vdim") or d)
    x = _rnd(h)
    q = _rnd(_rotated_unit(linear(x, W[p + "q"]).view(T, H, d), m.get("rot"), eps))
    if m.get("kv_from") is not None:
        k, v = shared[int(m["kv_from"])]
    else:
        k = _rnd(_rotated_unit(linear(x, W[p + "k"]).view(T, G, d), m.get("rot"), eps))
        v = _rnd(linear(x, W[p + "v"]).view(T, G, dv))
        if shared is not None:
            shared[index] = (k, v)
    per = H // G
    kh, vh = k.repeat_interleave(per, dim=1), v.repeat_interleave(per, dim=1)        # query head a reads kv head a // per
    scores = torch.einsum("ihd,jhd->hij", q, kh) * float(m["scale"])
    mask = m.get("mask")
    ok = visible(T, int(mask["size"]) if mask else None, int(mask.get("keep_first") or 0) if mask else 0)
    w = torch.softmax(scores.masked_fill(~ok[None], -math.inf), dim=-1)
    ctx = torch.einsum("hij,jhd->ihd", w, vh)
    ctx = _rnd(ctx) * torch.sigmoid(linear(x, W[p + "g"]))[:, :, None]               # one number per head
    return linear(_rnd(ctx).reshape(T, H * dv), W[p + "o"])


# ----------------------------------------------------------------------------- recurrences

def causal_filter(u: torch.Tensor, w: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """y_t = bias + sum_j w[:, j] u_(t - taps + 1 + j) per channel, zeros before the start; u [T, channels]."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=F), u])
    return sum(padded[j:j + u.shape[0]] * w[:, j].to(F) for j in range(taps)) + bias.to(F)


def fading_scan(q, k, v, g, dt, skip: float, S0=None):
    """One head. S_t = g_t S_(t-1) + dt_t k_t v_t^T, o_t = S_t^T q_t + skip v_t. q, k [T, N]; v [T, vdim]; g, dt [T]."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=F) if S0 is None else S0.clone()
    out = []
    for t in range(q.shape[0]):
        S = g[t] * S + dt[t] * k[t][:, None] * v[t][None, :]
        out.append(S.T @ q[t] + skip * v[t])
    return (torch.stack(out) if out else torch.zeros(0, v.shape[1], dtype=F)), S


def state_space(h, W, p: str, m: Mapping, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, dv, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m.get("groups") or 1)
    inner = H * dv
    rows = linear(_rnd(h), W[p + "in"])
    z, xbc, dt = rows[:, :inner], rows[:, inner:2 * inner + 2 * G * N], rows[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_filter(xbc, W[p + "conv"], W[p + "conv.b"]))
    xs = xbc[:, :inner].view(T, H, dv)
    B, C = xbc[:, inner:inner + G * N].view(T, G, N), xbc[:, inner + G * N:].view(T, G, N)
    dt = softplus(dt + W[p + "dt_bias"].to(F))
    g = torch.exp(-torch.exp(W[p + "A_log"].to(F)) * dt)
    per = H // G
    y = torch.stack([fading_scan(C[:, a // per], B[:, a // per], xs[:, a], g[:, a], dt[:, a], float(W[p + "D"][a]))[0]
                     for a in range(H)], dim=1).reshape(T, inner)
    n_groups = int(m.get("norm_groups") or 1)
    y = rms((y * silu(z)).view(T, n_groups, inner // n_groups), eps).reshape(T, inner) * W[p + "norm"].to(F)
    return linear(_rnd(y), W[p + "o"])


def memory_scan(q, k, v, i, f, S0=None, n0=None, m0: float = 0.0):
    """One head. m_t = max(f_t + m_(t-1), i_t); S_t = e^(f + m_(t-1) - m_t) S + e^(i - m_t) k v^T, n_t likewise with k alone;
    o_t = S_t^T q / (max(|n_t . q|, e^(-m_t)) + DENOMINATOR_FLOOR)."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=F) if S0 is None else S0.clone()
    n = torch.zeros(q.shape[1], dtype=F) if n0 is None else n0.clone()
    m = torch.tensor(float(m0), dtype=F)
    out = []
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep * S + write * k[t][:, None] * v[t][None, :]
        n = keep * n + write * k[t]
        m = new
        out.append(S.T @ q[t] / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + DENOMINATOR_FLOOR))
    return (torch.stack(out) if out else torch.zeros(0, v.shape[1], dtype=F)), S, n, m


def memory_gates(i_raw, f_raw, cap: float):
    """Log input and log forget gate from their projections (biases added)."""
    return cap * torch.tanh(i_raw / cap), log_sigmoid(cap * torch.tanh(f_raw / cap))


def matrix_memory(h, W, p: str, m: Mapping, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d = int(m["heads"]), int(m["dim"])
    dv = int(m.get("vdim") or d)
    x = _rnd(h)
    q = linear(x, W[p + "q"]).view(T, H, d) * d ** -0.5
    k, v = linear(x, W[p + "k"]).view(T, H, d), linear(x, W[p + "v"]).view(T, H, dv)
    i, f = memory_gates(linear(x, W[p + "i"]) + W[p + "i.b"].to(F), linear(x, W[p + "f"]) + W[p + "f.b"].to(F), float(m["gate_cap"]))
    o = torch.stack([memory_scan(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a])[0] for a in range(H)], dim=1)
    y = rms(o, eps).reshape(T, H * dv) * W[p + "norm"].to(F) * torch.sigmoid(linear(x, W[p + "g"]))
    return linear(_rnd(y), W[p + "o"])


# ----------------------------------------------------------------------------- feed-forward

def route_top(logits: torch.Tensor, top: int):
    """logits [T, E] -> (chosen [T, top], weights [T, top]): the largest logits (ties: the lower index), softmax over
    the chosen ones only; also the gap between the last chosen and the first refused logit."""
    order = torch.sort(logits, dim=-1, descending=True, stable=True)
    chosen, z = order.indices[:, :top], order.values[:, :top]
    gap = (order.values[:, top - 1] - order.values[:, top]) if logits.shape[1] > top else torch.full((logits.shape[0],), math.inf, dtype=F)
    return chosen, torch.softmax(z, dim=-1), gap


def routed_experts(h, W, p: str, f: Mapping, gaps: Optional[List] = None) -> torch.Tensor:
    x = _rnd(h)
    chosen, weights, gap = route_top(linear(x, W[p + "router"]), int(f["router"]["top"]))
    if gaps is not None:
        gaps.append(gap)
    out = torch.zeros_like(h)
    for e in range(int(f["router"]["experts"])):
        at = (chosen == e).nonzero()
        if not len(at):
            continue
        t, wt = at[:, 0], weights[at[:, 0], at[:, 1]]
        u = p + f"e{e}."
        hid = _rnd(silu(_rnd(linear(x[t], W[u + "gate"]))) * _rnd(linear(x[t], W[u + "up"])) * wt[:, None])
        out[t] += linear(hid, W[u + "down"])
    return out


# ----------------------------------------------------------------------------- the model

def forward(cfg: Mapping, W: Mapping[str, torch.Tensor], ids: Sequence[int], layer_outputs: Optional[List] = None,
            gaps: Optional[List] = None) -> torch.Tensor:
    """Logits [T, vocab] (float64) of one sequence; ``layer_outputs`` collects the stream after every layer,
    ``gaps`` every router's distance between the last chosen and the first refused logit, per position."""
    eps = float(cfg["norm"]["eps"])
    emb = cfg.get("embedding") or {}
    x = W["embed"].to(F)[torch.tensor(list(ids), dtype=torch.long)] * float(emb.get("scale", 1.0))
    shared: Dict[int, tuple] = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        n = norm(x, W[p + "norm1"], eps)
        if layer["type"] == "attention":
            y = windowed_attention(n, W, p + "mix.", m, eps, shared, i)
        elif layer["type"] == "mamba2":
            y = state_space(n, W, p + "mix.", m, eps)
        elif layer["type"] == "mlstm":
            y = matrix_memory(n, W, p + "mix.", m, eps)
        else:
            raise ValueError(f"unknown layer type {layer['type']!r}")
        out = x + y * W[p + "ls1"].to(F)
        if layer.get("mlp") is not None:
            out = out + routed_experts(n, W, p + "mlp.", layer["mlp"], gaps) * W[p + "ls2"].to(F)
        x = out
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return linear(_rnd(norm(x, W["final.norm"], eps)), W["head"])


def greedy(cfg: Mapping, W: Mapping[str, torch.Tensor], prompt: Sequence[int], n_new: int) -> List[int]:
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(torch.argmax(forward(cfg, W, ids)[-1])))
    return ids[len(prompt):]
