"""Tiny Bolelix configurations for the tests, random weights for them, and the comparison with the plain
implementation (plain_bolelix.py). The configurations differ from each other in every size and option and make
unequal what a model may happen to make equal (key and value sizes, kv heads and 1, groups and norm groups, the masks of a
layer and of the layers that read its keys, the order of the layer types, windows below and above a page or a key
chunk, kept first keys within and across pages, rotations over all or part of a head with and without a factor, routers
that choose one, some or all experts)."""
from __future__ import annotations

import copy
import functools
import json
from typing import Dict, List, Sequence, Tuple

import numpy as np
import torch

import helpers as H
import plain_bolelix as pb
from notirax_cases import CLUSTERS, _separated


def _att(heads, kv, dim, vdim, scale, mask, rot, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
         "mask": None if mask is None else {"size": mask[0], "keep_first": mask[1]},
         "rot": None if rot is None else {"base": rot[0], "dims": rot[1], "scaling": None if rot[2] is None else {"factor": rot[2]}}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _ssm(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def _mem(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def _moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def _base(vocab, width, eps, scale, layers):
    return {"architecture": "Bolelix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


CASES: Dict[str, dict] = {
    # a window of 24 that keeps 5 keys; two layers that read its keys, one through a wider window that keeps fewer, one
    # through a narrower window that keeps more; rotation over half a head
    "a": _base(200, 64, 1e-5, 2.0, [
        _layer("mamba2", _ssm(4, 16, 24, 2, 4, 2), _moe(6, 2, 24)),
        _layer("attention", _att(4, 2, 16, 16, 0.9, (24, 5), (1000.0, 8, 3.0)), _moe(5, 3, 40)),
        _layer("attention", _att(2, 2, 16, 16, 0.7, (40, 2), (1000.0, 8, 3.0), 1), _moe(4, 1, 32)),
        _layer("mlstm", _mem(3, 16, 24, 6.0), _moe(8, 4, 16)),
        _layer("attention", _att(6, 2, 16, 16, 0.8, (9, 11), (1000.0, 8, 3.0), 1), None)]),
    # nothing a multiple of eight; the memory first; a window of 33 keeping 18 (across a page border), read through no mask
    # at all; one of 5 keeping none; no rotation, rotation without a factor, over one pair; values of another size; filters
    # of one and two taps; one group and one norm group; layers without feed-forward; every expert and a single one
    "b": _base(97, 36, 3e-6, 1.0, [
        _layer("mlstm", _mem(3, 5, 9, 2.5), None),
        _layer("attention", _att(3, 1, 10, 7, 1.1, (33, 18), (50.0, 10, None)), _moe(4, 4, 10)),
        _layer("mamba2", _ssm(3, 7, 5, 1, 2, 1), _moe(9, 1, 5)),
        _layer("attention", _att(2, 2, 6, 9, 1.2, (5, 0), None), None),
        _layer("attention", _att(1, 1, 10, 7, 1.3, None, (50.0, 10, None), 1), _moe(5, 3, 7)),
        _layer("mamba2", _ssm(6, 3, 33, 3, 1, 2), None),
        _layer("attention", _att(1, 1, 13, 13, 0.9, (3, 1), (10000.0, 2, 0.5)), _moe(3, 2, 11)),
        _layer("mlstm", _mem(1, 33, 14, 20.0), _moe(2, 1, 9))]),
    # sizes that the tensor-core kernels take: keys and values of 64 and 128, a window of 150 keeping 40 (both across key
    # chunks of 128) read through one of 100 keeping 140, no mask at all, states of 128 x 64 and 64 x 128, a 16-row state
    "c": _base(256, 128, 2e-6, 4.0, [
        _layer("attention", _att(8, 2, 64, 64, 0.2, (150, 40), (30000.0, 32, 6.0)), _moe(8, 2, 32)),
        _layer("mamba2", _ssm(4, 64, 128, 2, 4, 1), _moe(4, 2, 64)),
        _layer("attention", _att(4, 2, 64, 64, 0.25, (100, 140), (30000.0, 32, 6.0), 0), None),
        _layer("mlstm", _mem(2, 64, 128, 15.0), _moe(16, 4, 16)),
        _layer("attention", _att(2, 1, 128, 128, 0.15, None, (500.0, 128, None)), _moe(3, 2, 64)),
        _layer("mamba2", _ssm(6, 24, 16, 3, 3, 4), _moe(3, 1, 24)),
        _layer("mlstm", _mem(3, 128, 40, 8.0), None)]),
}


def spec_of(cfg: dict):
    return H.spec_of(cfg)


def sharpened(cfg: dict, factor: float) -> dict:
    """The configuration with every attention scale times ``factor``: attention weights are peaked, a position's result
    hangs on single keys (the farthest its window still holds, a kept first key, a key hundreds of positions back), and a
    wrong key or a window one token off shows. (Queries and keys have a root mean square of one: the scale is what peaks.)"""
    cfg = copy.deepcopy(cfg)
    for l in cfg["layers"]:
        if l["type"] == "attention":
            l["mixer"]["scale"] *= factor
    return cfg


def make_weights(cfg: dict, seed: int, dtype=torch.bfloat16, decisive: bool = False) -> Dict[str, torch.Tensor]:
    """Random weights. With ``decisive`` (for bfloat16, where a close call may turn either way) tokens carry one of a few
    directions that the routers read, each router with well separated logits per direction."""
    from infer_b200.weights import random_weights
    W = random_weights(spec_of(cfg), seed, dtype)
    g = torch.Generator().manual_seed(seed)
    for i, l in enumerate(cfg["layers"]):
        for n, f in (("v", 6.0), ("o", 6.0), ("q", 3.0), ("k", 3.0), ("g", 10.0)) if l["type"] == "attention" else (("o", 4.0), ("g", 10.0)):
            if f"l{i}.mix.{n}" in W:                              # of a size that matters beside the other terms
                W[f"l{i}.mix.{n}"] = (W[f"l{i}.mix.{n}"].float() * f).to(dtype)
        if l["type"] == "mlstm":
            # A read-out is divided by its own size: where k.q of the one token that a state holds is nearly zero, its sign, and
            # with it the whole row's, hangs on the last bit. Keys that resemble queries keep k.q away from zero.
            W[f"l{i}.mix.k"] = (0.5 * W[f"l{i}.mix.k"].float() + W[f"l{i}.mix.q"].float()).to(dtype)
    embed = W["embed"].float() * 10.0
    if decisive:
        U = torch.linalg.qr(torch.randn(cfg["width"], CLUSTERS, generator=g)).Q.T         # [CLUSTERS, width]
        embed += 0.8 * cfg["width"] ** 0.5 * U[torch.arange(cfg["vocab"]) % CLUSTERS]
        for i, l in enumerate(cfg["layers"]):
            if l.get("mlp"):
                W[f"l{i}.mlp.router"] = (_separated(l["mlp"]["router"], g) @ U * (1.5 / cfg["width"] ** 0.5)).to(dtype)
    W["embed"] = embed.to(dtype)
    return W


def random_ids(cfg: dict, n: int, seed: int) -> List[int]:
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


@functools.lru_cache(maxsize=64)
def _oracle(cfg_json: str, seed: int, compute: str, ids: Tuple[int, ...], rounding: str):
    cfg = json.loads(cfg_json)
    W = H.as_compute(make_weights(cfg, seed, torch.bfloat16, compute == "bfloat16"), getattr(torch, compute))
    if rounding == "none":
        return pb.forward(cfg, W, list(ids)).numpy()
    with pb.rounded(getattr(torch, rounding)):
        return pb.forward(cfg, W, list(ids)).numpy()


def oracle(cfg: dict, seed: int, compute: torch.dtype, ids: Sequence[int], rounding=None) -> np.ndarray:
    n = lambda d: str(d).replace("torch.", "")
    return _oracle(json.dumps(cfg, sort_keys=True), seed, n(compute), tuple(int(i) for i in ids), "none" if rounding is None else n(rounding))


CLOSE_CALL = 0.05      # a router's gap between its last chosen and first refused logit below which bfloat16 roundings may turn the choice


@functools.lru_cache(maxsize=64)
def _router_gaps(cfg_json: str, seed: int, ids: Tuple[int, ...]) -> np.ndarray:
    cfg = json.loads(cfg_json)
    W = H.as_compute(make_weights(cfg, seed, torch.bfloat16, True), torch.bfloat16)
    gaps: List[torch.Tensor] = []
    pb.forward(cfg, W, list(ids), None, gaps)
    return torch.stack(gaps).min(dim=0).values.numpy() if gaps else np.full(len(ids), np.inf)


def clear_positions(cfg: dict, seed: int, ids: Sequence[int]) -> int:
    """Positions in front of the first one at which a router's choice is a close call."""
    gaps = _router_gaps(json.dumps(cfg, sort_keys=True), seed, tuple(int(i) for i in ids))
    close = np.nonzero(gaps < CLOSE_CALL)[0]
    return int(close[0]) if len(close) else len(ids)


OUTLIERS, OUTLIER_FACTOR = 0.02, 20.0


def _mostly_within(err: np.ndarray, bound: np.ndarray, what: str):
    """Every row within its bound, but for one row in fifty (at least one), which may be OUTLIER_FACTOR times over it. The
    memories and the gated norms divide a read-out by its own size: where it nearly vanishes (a query almost orthogonal to all
    that a state holds), a row's result hangs on the last bits of its inputs, in any implementation."""
    over = np.sort(err / bound)[::-1]
    allowed = max(1, int(OUTLIERS * len(over)))
    assert over[0] <= OUTLIER_FACTOR, f"{what}: row {int(np.argmax(err / bound))} is {over[0]:.1f} times over its bound"
    assert len(over) <= allowed or over[allowed] <= 1.0, f"{what}: {int((over > 1).sum())} of {len(over)} rows over their bounds"


def compare(got: np.ndarray, ref: np.ndarray, dtype: torch.dtype, what: str, ref_rounded=None, factor: float = 4.0):
    """float32: the largest difference of a row; bfloat16: a row's rms difference against the rounding noise that the plain
    implementation shows at that position (or on average, where that is larger)."""
    if dtype == torch.float32:
        _mostly_within(np.abs(got - ref).max(axis=-1), np.full(len(ref), H.F32_ATOL * max(1.0, float(np.abs(ref).max()))), what)
        return
    rms = lambda a: np.sqrt(np.mean(a ** 2, axis=-1))
    noise = max(float(rms((ref_rounded - ref).ravel())), 1e-3 * float(rms(ref.ravel())))
    _mostly_within(rms(got - ref), factor * np.maximum(rms(ref_rounded - ref), noise), what)


def check(cfg: dict, seed: int, dtype: torch.dtype, got: Dict[str, Dict[int, np.ndarray]], reqs: Dict[str, List[int]], what: str = ""):
    """The engine's rows against the plain implementation. In bfloat16, positions from the first one at which a
    router's choice is a close call are left out (the other expert is as right an answer there, and every later
    position reads what that one left in the caches and states). The float32 comparison leaves out nothing and is
    the sharp one; cuttings are compared bit by bit there."""
    for rid, ids in reqs.items():
        ref = oracle(cfg, seed, dtype, ids)
        rows = sorted(got[rid])
        if dtype != torch.float32:
            upto = clear_positions(cfg, seed, ids)
            rows = [p for p in rows if p < upto]
            if not rows:
                continue
        rounded = oracle(cfg, seed, dtype, ids, torch.bfloat16)[rows] if dtype != torch.float32 else None
        compare(np.stack([got[rid][p] for p in rows]), ref[rows], dtype, f"{what}/{rid}", rounded)
