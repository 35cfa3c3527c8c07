"""Matrix memory with exponential gates (the mLSTM of xLSTM).

Per head, with x the mixer's input row at a position:

    q = x Wq^T * dim^(-1/2),  k = x Wk^T          [dim]
    v = x Wv^T                                    [v_dim]
    i = cap tanh((x Wi^T + bi) / cap)             log input gate, one number
    f = log sigmoid(cap tanh((x Wf^T + bf) / cap))                  log forget gate, one number
    m' = max(f + m, i)                            a running maximum, 0 for a new request
    S <- e^(f + m - m') S + e^(i - m') k v^T      S [dim, v_dim], zero for a new request
    n <- e^(f + m - m') n + e^(i - m') k          n [dim], zero for a new request
    o = S^T q / (max(|n.q|, e^(-m')) + floor)

o is divided by its root mean square per head (eps inside the root); the heads are joined, multiplied by a weight per channel
and by sigmoid(x Wg^T), and projected by Wo.  S, n and m live in float32 in a state slot of the request and are carried from
step to step. All six projections are one matrix product with float32 result rows; gates, exponentials, the state and the norm
are float32 whatever the compute dtype.

``names`` renames the local tensors by role (q, k, v, gate, o, norm, input, input_bias, forget, forget_bias).
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..config.specs import PartSpec
from .base import Mixer, StateNeed, own_or_projected, register_mixer
from .linear import Linear

_NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "gate": "g_proj.weight", "o": "o_proj.weight",
          "norm": "norm.weight", "input": "i_gate.weight", "input_bias": "i_gate.bias", "forget": "f_gate.weight",
          "forget_bias": "f_gate.bias"}


def _names(spec: PartSpec):
    return {**_NAMES, **dict(spec.get("names") or {})}


@register_mixer("matrix_memory")
class MatrixMemory(Mixer):
    def __init__(self, spec: PartSpec, runtime):
        super().__init__(spec, runtime)
        self.hidden, self.n_heads, self.dim = int(spec["hidden_size"]), int(spec["num_heads"]), int(spec["head_dim"])
        self.v_dim = int(spec.get("v_head_dim") or self.dim)
        self.cap, self.floor, self.eps = float(spec["gate_cap"]), float(spec.get("floor", 1e-6)), float(spec["norm_eps"])
        if min(self.hidden, self.n_heads, self.dim, self.v_dim) <= 0 or self.eps <= 0 or self.cap <= 0 or self.floor < 0:
            raise ValueError("matrix_memory needs positive sizes, gate_cap and eps")
        if self.dim > ops.state_scan_max_dim():
            raise ValueError(f"a key size of {self.dim} is beyond what the recurrence kernel keeps in registers ({ops.state_scan_max_dim()})")
        self.proj: Optional[Linear] = None
        self.o: Optional[Linear] = None

    @classmethod
    def param_shapes(cls, spec):
        W, H, d = int(spec["hidden_size"]), int(spec["num_heads"]), int(spec["head_dim"])
        dv = int(spec.get("v_head_dim") or d)
        n = _names(spec)
        return {n["q"]: (H * d, W), n["k"]: (H * d, W), n["v"]: (H * dv, W), n["gate"]: (H * dv, W), n["o"]: (W, H * dv),
                n["norm"]: (H * dv,), n["input"]: (H, W), n["input_bias"]: (H,), n["forget"]: (H, W), n["forget_bias"]: (H,)}

    @classmethod
    def init_params(cls, spec, name, shape, gen):
        n = _names(spec)
        kw = dict(generator=gen, dtype=torch.float32, device=gen.device)
        if name == n["norm"]:
            return 1.0 + 0.1 * torch.randn(shape, **kw)
        if name == n["input_bias"]:
            return torch.randn(shape, **kw)
        if name == n["forget_bias"]:
            return 3.0 + torch.randn(shape, **kw)              # (most of a state survives a token)
        if name in (n["q"], n["k"], n["v"], n["input"], n["forget"]):
            return 0.3 * torch.randn(shape, **kw)
        return super().init_params(spec, name, shape, gen)

    def load(self, params):
        n = _names(self.spec)
        # result rows [q | k | v | gate | input gates | forget gates], float32, whole 16-byte pieces
        w = torch.cat([params[n[r]] for r in ("q", "k", "v", "gate", "input", "forget")], dim=0)
        self.proj = Linear(self.rt, torch.nn.functional.pad(w, (0, 0, 0, -w.shape[0] % 8)))
        f32 = dict(device=self.rt.device, dtype=torch.float32)
        self.norm_w, self.input_b, self.forget_b = (params[n[r]].to(**f32).contiguous() for r in ("norm", "input_bias", "forget_bias"))
        self.o = Linear(self.rt, params[n["o"]])

    def cache_need(self):
        return StateNeed({"S": ((self.n_heads, self.dim, self.v_dim), torch.float32), "n": ((self.n_heads, self.dim), torch.float32),
                          "m": ((self.n_heads,), torch.float32)})

    def input_product(self):
        return self.proj, "float32"

    def drop_input_product(self):
        self.proj = None

    def forward(self, x, step, cache, residual, write_cache=True):
        H, nq, nv = self.n_heads, self.n_heads * self.dim, self.n_heads * self.v_dim
        rows, c0 = own_or_projected(self, x, self.proj, torch.float32)
        gate_col = c0 + 2 * nq + nv
        gates = ops.memory_gates(rows, gate_col + nv, gate_col + nv + H, self.input_b, self.forget_b, self.cap, cache["m"], step, write_cache,
                                 blocks=self.rt.dtype == torch.bfloat16)
        o, den = ops.step_scan(rows, c0, c0 + nq, c0 + 2 * nq, gates, 0, H, 3 * H, cache["S"], step, H, 1, self.dim, self.v_dim, write_cache,
                               ones_state=cache["n"], chunked=self.rt.dtype == torch.bfloat16)
        # (the read-outs are linear in q: its constant is applied to them)
        y = ops.group_norm_gate(o, self.norm_w, self.eps, rows, gate_col, "sigmoid", H, self.v_dim, self.rt.dtype, den=den,
                                den_floor=gates, floor_col=2 * H, den_mult=float(self.dim) ** -0.5, den_eps=self.floor)
        if residual is None:
            return self.o(y, out_dtype=torch.float32)
        return self.o(y, residual=residual)
