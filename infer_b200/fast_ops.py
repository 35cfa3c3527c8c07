"""The fast kernels of the bfloat16 serving path (sm_100a): each function returns its result, or None
when the kernel does not take the shape, in which case the caller uses the plain kernel.

Kernels that need scratch memory (split-K partial tiles, flash-decoding partial results) share one
workspace per device, allocated once and grown on demand; calls on one stream run in order, so they
may share it (a registered side stream has its own).  One status word per device collects failures that kernels report (a page index out of
range, a bounded wait that ran out).
"""
from __future__ import annotations

import ctypes
import os
from typing import Dict, Optional

import torch

from . import ops
from .ops import KernelError, _call, _check, _fn, _ptr, _stream, c_float, c_int, c_int64, c_void_p, dtype_code


class DeviceState:
    """Per-device scratch shared by the fast kernels."""

    def __init__(self, device: torch.device):
        self.device = device
        self.status = torch.zeros(1, dtype=torch.int32, device=device)
        self.sm_count = torch.cuda.get_device_properties(device).multi_processor_count
        self._workspace = torch.empty(0, dtype=torch.float32, device=device)
        self._counters = torch.zeros(4096, dtype=torch.int32, device=device)
        self._retired = []

    def workspace(self, n_floats: int) -> torch.Tensor:
        if self._workspace.numel() < n_floats:
            if torch.cuda.is_current_stream_capturing():
                raise KernelError("the kernel workspace must be sized before a CUDA graph is captured")
            self._retired.append(self._workspace)        # captured graphs may still point at it
            self._workspace = torch.empty(max(n_floats, 1 << 22), dtype=torch.float32, device=self.device)
        return self._workspace

    def counters(self, n: int) -> torch.Tensor:
        if self._counters.numel() < n:
            if torch.cuda.is_current_stream_capturing():
                raise KernelError("the kernel counters must be sized before a CUDA graph is captured")
            self._retired.append(self._counters)
            self._counters = torch.zeros(max(n, 4096), dtype=torch.int32, device=self.device)
        return self._counters


_STATES: Dict[torch.device, DeviceState] = {}
_SIDE_STATES: Dict[tuple, DeviceState] = {}        # (device, raw handle of a registered side stream) -> its scratch


def register_side_stream(stream: "torch.cuda.Stream") -> None:
    """A stream on which a part runs kernels beside those of the step's own stream. Kernels launched while it is the
    current stream get a workspace and counters of their own (calls on ONE stream run in order and may share
    scratch; calls on two streams may not). The status word stays one per device."""
    device = torch.device("cuda", stream.device_index if hasattr(stream, "device_index") else stream.device.index)
    key = (device, stream.cuda_stream)
    if key not in _SIDE_STATES:
        st = DeviceState(device)
        st.status = device_state(device).status
        _SIDE_STATES[key] = st


def device_state(device) -> DeviceState:
    device = torch.device(device)
    if device.index is None:
        device = torch.device("cuda", torch.cuda.current_device())
    if _SIDE_STATES:
        side = _SIDE_STATES.get((device, torch._C._cuda_getCurrentRawStream(device.index)))
        if side is not None:
            return side
    st = _STATES.get(device)
    if st is None:
        st = _STATES[device] = DeviceState(device)
    return st


# ----------------------------------------------------------------------------- tensor-core GEMM

_PLAN_CACHE: Dict[tuple, Optional[tuple]] = {}


def gemm_plan(M: int, N: int, K: int, sm_count: int):
    """(swap, bn, splits, workspace floats, counters) for a product, or None if the kernel refuses the sizes."""
    key = (M, N, K, sm_count)
    if key not in _PLAN_CACHE:
        f = _fn("gemm", "ib_gemm_tc_plan", [c_int64, c_int64, c_int64, c_int] + [c_void_p] * 5)
        swap, bn, splits = ctypes.c_int(), ctypes.c_int(), ctypes.c_int()
        ws, nc = ctypes.c_int64(), ctypes.c_int64()
        rc = f(M, N, K, sm_count, ctypes.byref(swap), ctypes.byref(bn), ctypes.byref(splits), ctypes.byref(ws), ctypes.byref(nc))
        _PLAN_CACHE[key] = None if rc != 0 else (swap.value, bn.value, splits.value, ws.value, nc.value)
    return _PLAN_CACHE[key]


def gemm_tc(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, residual: Optional[torch.Tensor] = None,
            out_dtype: torch.dtype = torch.bfloat16, out: Optional[torch.Tensor] = None, plan=None,
            swiglu: bool = False) -> Optional[torch.Tensor]:
    """out = x @ w.T (+ bias) (+ residual) on the tcgen05 tensor cores; None if the sizes are refused.
    x [M, K], w [N, K] bfloat16; bias float32 [N]; residual float32 [M, N] (may be `out`). With ``swiglu`` the
    rows of w are gate/up features interleaved in blocks of 8 and the result is silu(gate) * up, [M, N/2]."""
    _check(x, "x", torch.bfloat16)
    _check(w, "w", torch.bfloat16)
    M, K = x.shape
    N = w.shape[0]
    if w.shape[1] != K:
        raise KernelError(f"gemm_tc: x is [{M},{K}] but w is {tuple(w.shape)}")
    st = device_state(x.device)
    plan = plan or gemm_plan(M, N, K, st.sm_count)
    if plan is None or (x.data_ptr() & 15) or (w.data_ptr() & 15) or (swiglu and N % 16):
        return None
    swap, bn, splits, ws_floats, n_counters = plan
    if bias is not None:
        _check(bias, "bias", torch.float32, (N,))
    if residual is not None:
        _check(residual, "residual", torch.float32, (M, N))
    n_out = N // 2 if swiglu else N
    if out is None:
        out = torch.empty((M, n_out), dtype=out_dtype, device=x.device)
    else:
        _check(out, "out", out_dtype, (M, n_out))
    # split-K of the swapped mapping goes through the cluster's shared memory and needs neither
    ws = st.workspace(ws_floats) if splits > 1 and ws_floats > 0 else None
    cnt = st.counters(n_counters) if splits > 1 and ws_floats > 0 else None
    f = _fn("gemm", "ib_gemm_tc", [c_void_p] * 5 + [c_int64] * 3 + [c_int] * 5 + [c_void_p] * 4)
    _call(f, x.data_ptr(), w.data_ptr(), _ptr(bias), _ptr(residual), out.data_ptr(), M, N, K, dtype_code(out_dtype),
          2 if swiglu else 0, swap, bn, splits, _ptr(ws), _ptr(cnt), st.status.data_ptr(), _stream())
    ops.note("gemm_tc:sliced_wide" if bn == 768 else "gemm_tc:persistent" if bn >= 256 else ("gemm_tc:swapped" if swap else "gemm_tc:one_tile"))
    return out


_SKINNY_LIMITS = None


def skinny_limits():
    """(most rows, longest row the fused norm takes) of the streaming kernel, as its library states them."""
    global _SKINNY_LIMITS
    if _SKINNY_LIMITS is None:
        f = _fn("gemvb", "ib_linear_skinny_bulk_limits", [c_void_p, c_void_p])
        rows, k = ctypes.c_int(), ctypes.c_int()
        f(ctypes.byref(rows), ctypes.byref(k))
        _SKINNY_LIMITS = (rows.value, k.value)
    return _SKINNY_LIMITS


def linear_skinny(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None,
                  residual: Optional[torch.Tensor] = None, out_dtype: torch.dtype = torch.bfloat16,
                  out: Optional[torch.Tensor] = None, swiglu: bool = False, cluster: int = 0,
                  norm_weight: Optional[torch.Tensor] = None, norm_eps: float = 0.0) -> Optional[torch.Tensor]:
    """The decode kernel: x [M <= 16, K] against w [N, K], weights streamed once; same epilogues as gemm_tc.
    With ``norm_weight`` x is the float32 residual stream and is RMS-normalised inside the kernel (rows up to
    ``skinny_limits()[1]`` long).
    cluster: CTAs sharing one tile's K range (0 = chosen by the kernel)."""
    fused = norm_weight is not None
    _check(x, "x", torch.float32 if fused else torch.bfloat16)
    _check(w, "w", torch.bfloat16)
    M, K = x.shape
    N = w.shape[0]
    if w.shape[1] != K:
        raise KernelError(f"linear_skinny: x is [{M},{K}] but w is {tuple(w.shape)}")
    max_rows, max_norm_k = skinny_limits()
    if M > max_rows or K % 8 or (x.data_ptr() & 15) or (w.data_ptr() & 15) or (swiglu and N % 16):
        return None
    if fused:
        _check(norm_weight, "norm_weight", torch.float32, (K,))
        if K > max_norm_k or (norm_weight.data_ptr() & 15):
            return None
    if bias is not None:
        _check(bias, "bias", torch.float32, (N,))
    if residual is not None:
        _check(residual, "residual", torch.float32, (M, N))
        out_dtype = torch.float32
    n_out = N // 2 if swiglu else N
    if out is None:
        out = torch.empty((M, n_out), dtype=out_dtype, device=x.device)
    else:
        _check(out, "out", out_dtype, (M, n_out))
    st = device_state(x.device)
    epi = 2 if swiglu else (1 if residual is not None else 0)
    f = _fn("gemvb", "ib_linear_skinny_bulk", [c_void_p, c_void_p, c_float] + [c_void_p] * 4 + [c_int64] * 3 + [c_int] * 4 +
            [c_void_p] * 2 + [c_int64, c_void_p])
    _call(f, x.data_ptr(), _ptr(norm_weight), float(norm_eps), w.data_ptr(), _ptr(bias), _ptr(residual), out.data_ptr(),
          M, N, K, dtype_code(out_dtype), epi, int(cluster), st.sm_count, st.status.data_ptr(), None, 0, _stream())
    return out


def linear(x, weight, bias, residual, out_dtype, out, swiglu=False):
    """The bfloat16 matrix product of the serving path: the streaming kernel for up to 16 rows, the tcgen05 kernel
    above that; None if neither takes the shape. x may be a DeferredNorm (the float32 residual stream plus the norm
    that is still to be applied): the streaming kernel then normalises inside, anything else materialises it."""
    from .parts.base import DeferredNorm
    if isinstance(x, DeferredNorm):
        if weight.dtype == torch.bfloat16 and x.h.shape[0] <= skinny_limits()[0]:
            y = linear_skinny(x.h, weight, bias, residual, out_dtype, out, swiglu, 0, x.norm.weight, x.norm.eps)
            if y is not None:
                return y
        x = x.materialize()
    if x.dtype != torch.bfloat16:
        return None
    if x.shape[0] <= skinny_limits()[0]:
        y = linear_skinny(x, weight, bias, residual, out_dtype, out, swiglu)
        if y is not None:
            return y
    return gemm_tc(x, weight, bias, residual, out_dtype, out, swiglu=swiglu)


GROUPED_FROM = 256            # tokens from which a routed feed-forward's rows are worth grouping by expert


def grouped_experts_worth(n_tokens: int, top: int, n_experts: int) -> bool:
    """True where the chosen experts' rows, each expert's padded to whole tiles, are well below tokens x experts."""
    return n_tokens >= GROUPED_FROM and 5 * (n_tokens * top + 64 * n_experts) <= 3 * n_tokens * n_experts


class RowGroups:
    """The rows of a step that each expert was chosen for, side by side (``ops``-level view of the grouping kernels): ``place`` int32
    [T, top], ``scale`` float32 [rows, 1] (the token's weight for the row's expert), the table of tiles."""

    def __init__(self, weights: torch.Tensor, chosen: torch.Tensor):
        _check(weights, "weights", torch.float32)
        _check(chosen, "chosen", torch.int32)
        self.T, self.top = chosen.shape
        self.E = weights.shape[1]
        tile = int(_fn("experts", "ib_group_tile_rows", [])())
        pairs = self.T * self.top
        self.max_tiles = pairs // tile + min(self.E, pairs)
        self.likely_tiles = min(self.max_tiles, -(-pairs // tile) + self.E // 2)
        self.rows = self.max_tiles * tile
        dev = weights.device
        self.place = torch.empty(pairs, dtype=torch.int32, device=dev)
        self.row_of = torch.empty(self.rows, dtype=torch.int32, device=dev)
        self.scale = torch.empty((self.rows, 1), dtype=torch.float32, device=dev)
        self.tiles = torch.empty(1 + self.max_tiles, dtype=torch.int32, device=dev)
        f = _fn("experts", "ib_group_rows", [c_void_p, c_void_p, c_int64, c_int, c_int] + [c_void_p] * 5)
        _call(f, chosen.data_ptr(), weights.data_ptr(), self.T, self.top, self.E, self.place.data_ptr(), self.row_of.data_ptr(),
              self.scale.data_ptr(), self.tiles.data_ptr(), _stream())

    def gather(self, x: torch.Tensor) -> torch.Tensor:
        """[rows, W]: x's row of each grouped row (zeros in the padding; rows of tiles that are not in use are left as they are)."""
        _check(x, "x", torch.bfloat16)
        out = torch.empty((self.rows, x.shape[1]), dtype=x.dtype, device=x.device)
        f = _fn("experts", "ib_gather_rows", [c_void_p, c_void_p, c_void_p, c_void_p, c_int64, c_int64, c_void_p])
        _call(f, x.data_ptr(), self.row_of.data_ptr(), self.tiles.data_ptr(), out.data_ptr(), self.rows, x.shape[1] * 2, _stream())
        return out

    def product(self, x: torch.Tensor, w: torch.Tensor, n_expert: int, halves: int, side: int, out_dtype: torch.dtype):
        """x [rows, K] times its expert's part of w. side 0: w [halves * E * n_expert, K] (an expert's rows of each half), result
        [rows, halves * padded], returned with padded; side 1: w [n_expert, E * K] (an expert's columns), result [rows, n_expert]."""
        _check(x, "x", torch.bfloat16)
        _check(w, "w", torch.bfloat16)
        K = x.shape[1]
        want = (halves * self.E * n_expert, K) if side == 0 else (n_expert, self.E * K)
        if x.shape[0] != self.rows or tuple(w.shape) != want:
            raise KernelError(f"grouped product: x {tuple(x.shape)}, w {tuple(w.shape)}, expected {self.rows} rows and {want}")
        st = device_state(x.device)
        f = _fn("gemm", "ib_gemm_tc_grouped", [c_void_p] * 3 + [c_int64] * 4 + [c_int] * 3 + [c_void_p, c_int, c_int, c_void_p, c_void_p, c_void_p])
        padded = ctypes.c_int64(0)
        args = [self.max_tiles, self.likely_tiles, n_expert, K, self.E, halves, side, self.tiles.data_ptr(), dtype_code(out_dtype), st.sm_count,
                st.status.data_ptr(), ctypes.addressof(padded), _stream()]
        if f(None, w.data_ptr(), None, *args):
            raise KernelError("grouped product: " + f._lib.ib_last_error().decode())
        out = torch.empty((self.rows, halves * padded.value), dtype=out_dtype, device=x.device)
        _call(f, x.data_ptr(), w.data_ptr(), out.data_ptr(), *args)
        return out, padded.value

    def combine(self, y: torch.Tensor, residual: Optional[torch.Tensor] = None) -> torch.Tensor:
        """float32 [T, W]: (residual +) the sum of each token's rows, over ``residual`` where given."""
        _check(y, "y", torch.float32)
        W = y.shape[1]
        out = residual if residual is not None else torch.empty((self.T, W), dtype=torch.float32, device=y.device)
        f = _fn("experts", "ib_combine_rows", [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int64, c_int64, c_void_p])
        _call(f, y.data_ptr(), self.place.data_ptr(), self.top, _ptr(residual), out.data_ptr(), self.T, W, _stream())
        return out


def attention_supported(n_heads: int, n_kv: int, head_dim: int, page_size: int) -> bool:
    return head_dim % 16 == 0 and 16 <= head_dim <= 128 and page_size == 16 and n_heads // n_kv <= 16


ATTENTION_MAX_CLUSTERS = 32       # clusters of 8 slices per (segment, kv head), for long contexts at small batches
ATTENTION_CLUSTER_PAGES = 16      # pages a slice keeps at least when a (segment, kv head) gets several clusters
ATTENTION_CLUSTER_FROM = 96       # ... which it gets when one cluster's slices would each walk at least this many pages


def _decode_splits(st, n_decode: int, n_kv: int, visible: int):
    """(slices per cluster, clusters per (segment, kv head)). Slices: a power of two up to 8, enough CTAs for about
    one per SM, and at least 8 pages (two per warp) in a slice. Clusters: more than one only for long contexts (the
    second level costs about 5 us per layer: measured at batch 8 it loses at 8,192 tokens, 1.56 against 1.44 ms per
    step, and wins at 30,000, 2.50 against 2.78; at batch 1 and 30,000 tokens 1.41 against 2.21), then as many as keep
    16 pages (four per warp) in a slice, up to two CTAs per SM."""
    units = max(1, n_decode * n_kv)
    pages = max(1, -(-visible // 16))
    n = 1
    # (with nearly a CTA per SM already, two slices do not pay for their merge: 25.1 against 26.2 us at batch 64)
    while n < 8 and units * n < st.sm_count and pages // (2 * n) >= 8 and not (n == 1 and 6 * units >= 5 * st.sm_count):
        n *= 2
    clusters = 1
    if n == 8 and pages >= 8 * ATTENTION_CLUSTER_FROM:
        clusters = max(1, min(pages // (8 * ATTENTION_CLUSTER_PAGES), (2 * st.sm_count) // (units * 8), ATTENTION_MAX_CLUSTERS))
    return n, clusters


def _decode_scratch(st, n_segments: int, n_kv: int, head_dim: int, clusters: int):
    """Workspace and counters for several clusters per (segment, kv head); (None, None) for one."""
    if clusters <= 1:
        return None, None
    return st.workspace(n_segments * n_kv * clusters * (16 * head_dim + 32)), st.counters(n_segments * n_kv)


# The prefill kernel on tcgen05 / tensor memory (attention_tc.cu) serves head sizes 64 and 128; INFER_B200_ATTN_TC=0
# leaves prefill to the mma.sync kernel.
ATTENTION_TC = os.environ.get("INFER_B200_ATTN_TC", "1") == "1"
ATTENTION_TC_HEAD_DIMS = (64, 128)
# Sharing a query tile's keys among CTAs (INFER_B200_ATTN_TC_SPLIT=1 switches it off): the kernel's limits.
ATTENTION_TC_MAX_SPLIT = int(os.environ.get("INFER_B200_ATTN_TC_SPLIT", "4"))
ATTENTION_TC_PART_MIN_TILES = 4


def prefill_split(sm_count: int, n_heads: int, n_prefill: int, max_q_len: int, max_ctx_len: int, window: Optional[int]) -> int:
    """Into how many parts the tcgen05 prefill kernel may cut the keys of a query tile. One CTA serves 128 queries of a
    head and walks over their keys in tiles of 128; it has an SM to itself, and starting and finishing a CTA costs
    about as much as three key tiles. So keys are shared only while all CTAs still run at once (a portion behind a
    long context on few heads: 48 CTAs of 36 key tiles become 144 of 12); with more CTAs than SMs the extra starts
    cost more than the evening-out gains (measured at 2,048 tokens on 12 heads: 38.5 us whole, 42 us shared)."""
    if n_prefill <= 0 or max_q_len <= 1:
        return 1
    ctx0 = max_ctx_len - max_q_len
    key_tiles = []
    for q_first in range(ctx0, max_ctx_len, 128):
        q_last = min(max_ctx_len - 1, q_first + 127)
        lo = max(0, q_first - window + 1) if window else 0
        key_tiles.append(q_last // 128 - lo // 128 + 1)
    if max(key_tiles) < 2 * ATTENTION_TC_PART_MIN_TILES:
        return 1
    for split in range(ATTENTION_TC_MAX_SPLIT, 1, -1):
        ctas = n_heads * n_prefill * sum(max(1, min(split, n // ATTENTION_TC_PART_MIN_TILES)) for n in key_tiles)
        if ctas <= sm_count:
            return split
    return 1


def attention_fast(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor,
                   seg_start: torch.Tensor, seg_pos0: torch.Tensor, n_heads: int, n_kv: int, head_dim: int,
                   window: Optional[int], scale: float, has_decode: bool, max_q_len: int, max_ctx_len: int,
                   n_decode: Optional[int] = None, n_splits: Optional[int] = None, n_clusters: int = 1,
                   tc_split: Optional[int] = None) -> Optional[torch.Tensor]:
    """Tensor-core attention of a step's segments over the paged bfloat16 cache; None if the shape is refused.
    The library is compiled for this head size at first use."""
    n_pages, ckv, page_size, chd = k_cache.shape
    if q.dtype != torch.bfloat16 or not attention_supported(n_heads, n_kv, head_dim, page_size):
        return None
    _check(q, "q", torch.bfloat16)
    T = q.shape[0]
    _check(q, "q", None, (T, n_heads * head_dim))
    _check(k_cache, "k_cache", torch.bfloat16)
    _check(v_cache, "v_cache", torch.bfloat16, k_cache.shape)
    if ckv != n_kv or chd != head_dim:
        raise KernelError(f"cache shape {tuple(k_cache.shape)} does not match kv_heads={n_kv}, head_dim={head_dim}")
    S = seg_pos0.numel()
    _check(seg_start, "seg_start", torch.int32, (S + 1,))
    _check(seg_pos0, "seg_pos0", torch.int32, (S,))
    _check(block_table, "block_table", torch.int32)
    st = device_state(q.device)
    if n_splits is None:
        visible = min(max_ctx_len, window) if window else max_ctx_len
        n_splits, n_clusters = _decode_splits(st, n_decode if n_decode is not None else S, n_kv, visible) if has_decode else (1, 1)
    ws, cnt = _decode_scratch(st, S, n_kv, head_dim, n_clusters)
    out = torch.empty_like(q)
    # Segments of two or more tokens go to the tcgen05 kernel where it takes the head size; one-token segments, and
    # everything else, to the mma.sync kernels (a call with max_q_len = 1 launches no prefill kernel).
    tc = ATTENTION_TC and max_q_len > 1 and head_dim in ATTENTION_TC_HEAD_DIMS and page_size == 16
    if tc:
        g = _fn("attn_tc", "ib_attention_prefill_tc", [c_void_p] * 5 + [c_int] + [c_void_p] * 2 + [c_int, c_int64] + [c_int] * 5 +
                [c_float, c_int64, c_int] + [c_void_p] * 2 + [c_int, c_void_p, c_int64, c_void_p, c_int64, c_int], {"IB_HEAD_DIM": head_dim})
        n_prefill = S - (n_decode or 0)
        split = prefill_split(st.sm_count, n_heads, n_prefill, max_q_len, max_ctx_len, window) if tc_split is None else tc_split
        tc_ws = tc_cnt = None
        if split > 1:
            tiles = max(1, n_prefill) * n_heads * -(-max_q_len // 128)
            tc_ws, tc_cnt = st.workspace(tiles * split * (128 * head_dim + 256)), st.counters(tiles)
            ops.note("attention_prefill_tc:shared_query_tiles")
        _call(g, q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), block_table.data_ptr(),
              block_table.shape[1], seg_start.data_ptr(), seg_pos0.data_ptr(), S, T, n_heads, n_kv, head_dim, page_size,
              int(window or 0), float(scale), n_pages, int(max_q_len), st.status.data_ptr(), _stream(), int(split),
              _ptr(tc_ws), 0 if tc_ws is None else tc_ws.numel(), _ptr(tc_cnt), 0 if tc_cnt is None else tc_cnt.numel(),
              int(n_prefill) if n_decode is not None else 0)
        if max_q_len > 128:
            ops.note("attention_prefill_tc:several_query_tiles")
        if not has_decode:
            return out
    f = _fn("attn", "ib_attention_fast", [c_void_p] * 5 + [c_int] + [c_void_p] * 2 + [c_int] * 6 + [c_float, c_int64] +
            [c_int] * 3 + [c_void_p] * 2 + [c_int] + [c_void_p] * 2, {"IB_HEAD_DIM": head_dim})
    _call(f, q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), block_table.data_ptr(),
          block_table.shape[1], seg_start.data_ptr(), seg_pos0.data_ptr(), S, n_heads, n_kv, head_dim, page_size,
          int(window or 0), float(scale), n_pages, int(has_decode), 1 if tc else int(max_q_len), int(n_splits),
          st.status.data_ptr(), _stream(), int(n_clusters), _ptr(ws), _ptr(cnt))
    return out


def attention_prefill_biased(q, k_cache, v_cache, block_table, step, n_heads, n_kv, head_dim, window, scale,
                             bias_by_head: Optional[torch.Tensor], sink: Optional[torch.Tensor], keep_first: int = 0,
                             slopes: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    """The tcgen05 prefill kernel with a bias per (head, distance) (float32 [heads, L], already divided by the scale),
    a sink per head, kept first keys (with a window: every query also sees the keys below ``keep_first``) and a slope
    per head (float32 [heads]: slope * distance is taken off the scaled score), on the segments of two or more tokens;
    the rows of one-token segments are left unwritten. None if the shape is refused."""
    n_pages, ckv, page_size, chd = k_cache.shape
    if (q.dtype != torch.bfloat16 or not ATTENTION_TC or head_dim not in ATTENTION_TC_HEAD_DIMS or page_size != 16
            or not attention_supported(n_heads, n_kv, head_dim, page_size) or not scale > 0):
        return None
    T = q.shape[0]
    _check(q, "q", torch.bfloat16, (T, n_heads * head_dim))
    _check(k_cache, "k_cache", torch.bfloat16, (n_pages, n_kv, page_size, head_dim))
    _check(v_cache, "v_cache", torch.bfloat16, k_cache.shape)
    if bias_by_head is not None:
        _check(bias_by_head, "bias_by_head", torch.float32)
        if bias_by_head.dim() != 2 or bias_by_head.shape[0] != n_heads:
            raise KernelError(f"bias_by_head must be [{n_heads}, distances], got {tuple(bias_by_head.shape)}")
    if sink is not None:
        _check(sink, "sink", torch.float32, (n_heads,))
    if slopes is not None:
        _check(slopes, "slopes", torch.float32, (n_heads,))
    S = step.seg_pos0.numel()
    st = device_state(q.device)
    n_prefill = sum(1 for n in step.seg_lens if n > 1)
    split = prefill_split(st.sm_count, n_heads, n_prefill, step.max_q_len, step.max_ctx_len, window)
    tc_ws = tc_cnt = None
    if split > 1:
        tiles = max(1, n_prefill) * n_heads * -(-step.max_q_len // 128)
        tc_ws, tc_cnt = st.workspace(tiles * split * (128 * head_dim + 256)), st.counters(tiles)
    out = torch.empty_like(q)
    keep_first = int(keep_first or 0) if window else 0
    kept = keep_first > 0 or slopes is not None                 # (the entry point that takes them; the other is unchanged)
    sig = [c_void_p] * 5 + [c_int] + [c_void_p] * 2 + [c_int, c_int64] + [c_int] * 5 + [c_float, c_int64, c_int] + [c_void_p] * 2 + \
          [c_int, c_void_p, c_int64, c_void_p, c_int64, c_int, c_void_p, c_int, c_void_p]
    g = _fn("attn_tc", "ib_attention_prefill_tc_kept" if kept else "ib_attention_prefill_tc_biased", sig + ([c_int, c_void_p] if kept else []),
            {"IB_HEAD_DIM": head_dim})
    args = [q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), block_table.data_ptr(), block_table.shape[1],
            step.seg_start.data_ptr(), step.seg_pos0.data_ptr(), S, T, n_heads, n_kv, head_dim, page_size, int(window or 0), float(scale),
            n_pages, int(step.max_q_len), st.status.data_ptr(), _stream(), int(split), _ptr(tc_ws), 0 if tc_ws is None else tc_ws.numel(),
            _ptr(tc_cnt), 0 if tc_cnt is None else tc_cnt.numel(), int(n_prefill), _ptr(bias_by_head),
            0 if bias_by_head is None else bias_by_head.shape[1], _ptr(sink)]
    _call(g, *(args + ([keep_first, _ptr(slopes)] if kept else [])))
    return out


# Attention whose heads exchange their scores (talk_prefill.cu): sizes that the tensor-core kernels are built for, and how
# much memory a launch's scores may take (a launch covers as many query tiles of 128 tokens as fit).
TALK_PREFILL_DIMS, TALK_PREFILL_MAX_HEADS = (64, 128), 32
TALK_SCORES_MAX_BYTES = 512 << 20


def talk_key_tiles(max_ctx_len: int, window: Optional[int], chunk: Optional[int]) -> int:
    """The most key tiles of 128 (aligned to absolute positions) that 128 neighbouring queries see."""
    n = -(-max_ctx_len // 128)
    seen = min([int(v) for v in (window, chunk) if v], default=None)
    if seen is not None:
        n = min(n, (seen + 127 + 126) // 128 + 1)
    return max(1, n)


TALK_START_BLOCKS = 2             # what starting a CTA of the score kernel costs, in blocks of 16 queries (of eight a query tile has)


def talk_q_split(sm_count: int, lens, max_ctx_len: int, window: Optional[int], chunk: Optional[int], qt0: int, n_qt: int) -> int:
    """How many CTAs share a (query tile, key tile) pair of the score kernel: rounds over the SMs times the time of a CTA.
    Counts the pairs of portions that end at max_ctx_len (captured steps know no more); any answer is correct."""
    pairs = 0
    for m in lens:
        for qt in range(qt0, min(qt0 + n_qt, -(-m // 128))):
            first = max_ctx_len - m + 128 * qt
            lo = max([0] + ([first - window + 1] if window else []) + ([first // chunk * chunk] if chunk else []))
            pairs += min(max_ctx_len - 1, first + 127) // 128 - lo // 128 + 1
    return min((1, 2, 4), key=lambda s: -(-max(1, pairs) * s // sm_count) * (TALK_START_BLOCKS + 8 / s))


def talk_attention_prefill(q: torch.Tensor, q_col: int, k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor, step,
                           n_heads: int, n_kv: int, head_dim: int, v_head_dim: int, window: Optional[int], chunk: Optional[int],
                           scale: float, cap: float, talk: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
    """``ops.talk_attention`` of the step's segments of two or more tokens on the tensor cores; the rows of one-token
    segments are left unwritten. None if the shape is refused. The library is compiled for these sizes at first use."""
    if not ATTENTION_TC or head_dim not in TALK_PREFILL_DIMS or v_head_dim not in TALK_PREFILL_DIMS or n_heads > TALK_PREFILL_MAX_HEADS:
        return None
    T, ld, n_pages, page_size = ops._check_talk(q, q_col, k_cache, v_cache, block_table, n_heads, n_kv, head_dim, v_head_dim, talk)
    if q.dtype != torch.bfloat16 or q_col % 8 or ld % 8 or page_size != 16:
        return None
    defines = {"IB_HEAD_DIM": head_dim, "IB_V_DIM": v_head_dim, "IB_HEADS": n_heads}
    if not _fn("talk_pf", "ib_talk_prefill_fits", [c_int] * 5, defines)(n_heads, n_kv, head_dim, v_head_dim, page_size):
        return None
    st = device_state(q.device)
    n_long = sum(1 for n in step.seg_lens if n > 1)
    tiles = talk_key_tiles(step.max_ctx_len, window, chunk)
    n_qt = -(-step.max_q_len // 128)
    per_qt = n_long * n_heads * tiles * 128 * 128
    at_once = max(1, min(n_qt, TALK_SCORES_MAX_BYTES // (4 * per_qt)))
    scores = torch.empty(per_qt * at_once, dtype=torch.float32, device=q.device)
    out = torch.empty((T, n_heads * v_head_dim), dtype=q.dtype, device=q.device)
    f = _fn("talk_pf", "ib_talk_prefill", [c_void_p, c_int64, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int,
                                           c_int64] + [c_int] * 7 + [c_float, c_float, c_void_p, c_int64] + [c_int] * 4 +
            [c_void_p, c_int64, c_int, c_void_p, c_void_p], defines)
    for qt0 in range(0, n_qt, at_once):
        n = min(at_once, n_qt - qt0)
        q_split = talk_q_split(st.sm_count, [m for m in step.seg_lens if m > 1], step.max_ctx_len, window, chunk, qt0, n)
        _call(f, q.data_ptr(), ld, int(q_col), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), block_table.data_ptr(),
              block_table.shape[1], step.seg_start.data_ptr(), step.seg_pos0.data_ptr(), step.seg_pos0.numel(), T, n_heads, n_kv, head_dim,
              v_head_dim, page_size, int(window or 0), int(chunk or 0), float(scale), float(cap or 0.0), _ptr(talk), n_pages, qt0, n, tiles,
              q_split, scores.data_ptr(), scores.numel(), n_long, st.status.data_ptr(), _stream())
    return out


def decode_fused_supported(n_heads: int, n_kv: int, head_dim: int, page_size: int) -> bool:
    return attention_supported(n_heads, n_kv, head_dim, page_size) and head_dim % 32 == 0


def attention_decode_fused(qkv: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, k_cache: torch.Tensor,
                           v_cache: torch.Tensor, block_table: torch.Tensor, seg_start: torch.Tensor,
                           seg_pos0: torch.Tensor, n_heads: int, n_kv: int, head_dim: int, window: Optional[int],
                           scale: float, max_ctx_len: int, write_cache: bool = True,
                           n_splits: Optional[int] = None, n_clusters: int = 1) -> Optional[torch.Tensor]:
    """Decode-only steps: rotation of q and k, the cache write of the new positions and attention in ONE kernel.
    qkv [S, (heads + 2 kv) * head_dim] packed rows with the bias added. Returns [S, heads * head_dim]."""
    n_pages, ckv, page_size, chd = k_cache.shape
    if qkv.dtype != torch.bfloat16 or not decode_fused_supported(n_heads, n_kv, head_dim, page_size):
        return None
    S = seg_pos0.numel()
    _check(qkv, "qkv", torch.bfloat16, (S, (n_heads + 2 * n_kv) * head_dim))
    _check(k_cache, "k_cache", torch.bfloat16)
    _check(v_cache, "v_cache", torch.bfloat16, k_cache.shape)
    if ckv != n_kv or chd != head_dim:
        raise KernelError(f"cache shape {tuple(k_cache.shape)} does not match kv_heads={n_kv}, head_dim={head_dim}")
    _check(cos, "cos", torch.float32)
    _check(sin, "sin", torch.float32, cos.shape)
    if cos.shape[1] != head_dim // 2:
        raise KernelError("rotary tables must be [max_positions, head_dim/2]")
    _check(seg_start, "seg_start", torch.int32, (S + 1,))
    _check(seg_pos0, "seg_pos0", torch.int32, (S,))
    _check(block_table, "block_table", torch.int32)
    st = device_state(qkv.device)
    if n_splits is None:
        visible = min(max_ctx_len, window) if window else max_ctx_len
        n_splits, n_clusters = _decode_splits(st, S, n_kv, visible)
    ws, cnt = _decode_scratch(st, S, n_kv, head_dim, n_clusters)
    out = torch.empty((S, n_heads * head_dim), dtype=torch.bfloat16, device=qkv.device)
    f = _fn("attn", "ib_attention_decode_fused", [c_void_p] * 7 + [c_int] + [c_void_p] * 2 + [c_int] * 6 + [c_float, c_int64] +
            [c_int] * 2 + [c_void_p] * 2 + [c_int64, c_void_p] + [c_int] + [c_void_p] * 2, {"IB_HEAD_DIM": head_dim})
    _call(f, qkv.data_ptr(), cos.data_ptr(), sin.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(),
          block_table.data_ptr(), block_table.shape[1], seg_start.data_ptr(), seg_pos0.data_ptr(), S, n_heads, n_kv,
          head_dim, page_size, int(window or 0), float(scale), n_pages, int(write_cache), int(n_splits),
          st.status.data_ptr(), None, 0, _stream(), int(n_clusters), _ptr(ws), _ptr(cnt))
    return out


def attention(q, cache, table, step, n_heads, n_kv, head_dim, window, scale):
    n_decode = sum(1 for n in step.seg_lens if n == 1)
    return attention_fast(q, cache.k, cache.v, table, step.seg_start, step.seg_pos0, n_heads, n_kv, head_dim, window,
                          scale, n_decode > 0, step.max_q_len, step.max_ctx_len, n_decode)


def gate_up_swiglu(x, gate_up_weight):
    """silu(x Wg^T) * (x Wu^T) in one kernel; gate_up_weight rows interleaved in blocks of 8."""
    return linear(x, gate_up_weight, None, None, torch.bfloat16, None, swiglu=True)
