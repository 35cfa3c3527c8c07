"""State space layer with a matrix state per head that fades by one number per head and token (Mamba-2).

With x the mixer's input row at a position, ``num_heads`` heads of values of size v_dim (inner = num_heads * v_dim),
``groups`` groups of state vectors of size N = ``state_size`` (head h uses group h // (num_heads / groups)):

    [z (inner) | u (inner) | B (groups x N) | C (groups x N) | r (num_heads)] = W_in x
    [v | k | q] = silu(filter([u | B | C]))      one short causal filter over time per channel, with a bias; zeros before
                                                 the sequence
    dt = softplus(r + dt_bias),   g = exp(-exp(A_log) dt)                              per head
    S <- g S + dt k v^T;   o = S^T q + D v                                             S [N, v_dim], zero for a new request
    y = o * silu(z), divided by its root mean square in ``norm_groups`` equal parts (eps inside the root), times a weight per
    channel; output product.

S (float32) and the filter's last taps - 1 inputs (float32) are the request's state. The input product has float32 result
rows; steps, decays, their exponentials, the state and the norm are float32 whatever the compute dtype.

``names`` renames the local tensors by role (in, filter, filter_bias, dt_bias, a_log, skip, norm, o).
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..config.specs import PartSpec
from .base import Mixer, StateNeed, own_or_projected, register_mixer
from .linear import Linear

_NAMES = {"in": "in_proj.weight", "filter": "filter.weight", "filter_bias": "filter.bias", "dt_bias": "dt_bias", "a_log": "A_log",
          "skip": "D", "norm": "norm.weight", "o": "o_proj.weight"}


def _names(spec: PartSpec):
    return {**_NAMES, **dict(spec.get("names") or {})}


def _sizes(spec: PartSpec):
    """(width, heads, value size, state size, groups, filter taps, inner channels, filtered channels)."""
    W, H, dv, N = (int(spec[k]) for k in ("hidden_size", "num_heads", "v_head_dim", "state_size"))
    G, taps = int(spec.get("groups") or 1), int(spec.get("filter_taps") or 1)
    return W, H, dv, N, G, taps, H * dv, H * dv + 2 * G * N


@register_mixer("state_space")
class StateSpace(Mixer):
    def __init__(self, spec: PartSpec, runtime):
        super().__init__(spec, runtime)
        self.hidden, self.n_heads, self.v_dim, self.state, self.groups, self.taps, self.inner, self.channels = _sizes(spec)
        self.norm_groups, self.eps = int(spec.get("norm_groups") or 1), float(spec["norm_eps"])
        if min(self.hidden, self.n_heads, self.v_dim, self.state, self.groups, self.taps, self.norm_groups) <= 0 or self.eps <= 0:
            raise ValueError("state_space needs positive sizes and eps")
        if self.n_heads % self.groups or self.inner % self.norm_groups:
            raise ValueError(f"state_space: {self.n_heads} heads in {self.groups} groups, {self.inner} channels in {self.norm_groups} norm groups")
        if self.state > ops.state_scan_max_dim():
            raise ValueError(f"a state of {self.state} rows is beyond what the recurrence kernel keeps in registers ({ops.state_scan_max_dim()})")
        self.proj: Optional[Linear] = None
        self.o: Optional[Linear] = None

    @classmethod
    def param_shapes(cls, spec):
        W, H, dv, N, G, taps, inner, channels = _sizes(spec)
        n = _names(spec)
        return {n["in"]: (inner + channels + H, W), n["filter"]: (channels, taps), n["filter_bias"]: (channels,), n["dt_bias"]: (H,),
                n["a_log"]: (H,), n["skip"]: (H,), n["norm"]: (inner,), n["o"]: (W, inner)}

    @classmethod
    def init_params(cls, spec, name, shape, gen):
        n = _names(spec)
        kw = dict(generator=gen, dtype=torch.float32, device=gen.device)
        if name == n["filter"]:
            w = 0.3 * torch.randn(shape, **kw)
            w[:, -1] += 1.0
            return w
        if name == n["filter_bias"]:
            return 0.2 * torch.randn(shape, **kw)
        if name in (n["norm"], n["skip"]):
            return 1.0 + 0.1 * torch.randn(shape, **kw)
        if name == n["a_log"]:
            return torch.log(0.1 + 2.0 * torch.rand(shape, **kw))
        if name == n["dt_bias"]:
            return torch.randn(shape, **kw) - 2.0
        if name == n["in"]:
            return 0.3 * torch.randn(shape, **kw)
        return super().init_params(spec, name, shape, gen)

    def load(self, params):
        n = _names(self.spec)
        w = params[n["in"]]                                   # result rows [z | u | B | C | r], float32, whole 16-byte pieces
        self.proj = Linear(self.rt, torch.nn.functional.pad(w, (0, 0, 0, -w.shape[0] % 8)))
        f32 = dict(device=self.rt.device, dtype=torch.float32)
        self.filter_w = params[n["filter"]].to(**f32).t().contiguous()                  # tap-major [taps, channels]
        self.filter_b, self.dt_bias, self.a_log, self.skip, self.norm_w = (
            params[n[r]].to(**f32).contiguous() for r in ("filter_bias", "dt_bias", "a_log", "skip", "norm"))
        self.o = Linear(self.rt, params[n["o"]])

    def cache_need(self):
        shapes = {"S": ((self.n_heads, self.state, self.v_dim), torch.float32)}
        if self.taps > 1:
            shapes["tails"] = ((self.taps - 1, self.channels), torch.float32)
        return StateNeed(shapes)

    def input_product(self):
        return self.proj, "float32"

    def drop_input_product(self):
        self.proj = None

    def forward(self, x, step, cache, residual, write_cache=True):
        rows, c0 = own_or_projected(self, x, self.proj, torch.float32)
        u_col = c0 + self.inner
        tails = cache.get("tails")
        # with one token per request, the thread that filters a channel is the only reader of its tail and moves it too
        inline_tail = tails is not None and write_cache and step.max_q_len == 1
        prep, g_col = ops.filter_prepare(rows, u_col, self.filter_w, self.filter_b, tails, u_col + self.channels, self.dt_bias,
                                         self.a_log, step, inline_tail)
        if tails is not None and write_cache and not inline_tail:
            ops.tail_update(rows, u_col, tails, step.seg_start, step.seg_slot)
        k_col = self.inner
        q_col = k_col + self.groups * self.state
        o = ops.step_scan(prep, q_col, k_col, 0, prep, g_col, g_col + self.n_heads, g_col + 2 * self.n_heads, cache["S"], step, self.n_heads,
                          self.n_heads // self.groups, self.state, self.v_dim, write_cache, skip=self.skip,
                          chunked=self.rt.dtype == torch.bfloat16)
        y = ops.group_norm_gate(o, self.norm_w, self.eps, rows, c0, "silu", self.norm_groups, self.inner // self.norm_groups,
                                self.rt.dtype, gate_first=True)
        if residual is None:
            return self.o(y, out_dtype=torch.float32)
        return self.o(y, residual=residual)
