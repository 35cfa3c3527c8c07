"""Tiny Notirax configurations for the tests, random weights for them, and the comparison with the plain
implementation (plain_notirax.py). The configurations differ from each other in every size and option and make unequal
what a model may happen to make equal (key and value sizes, heads and kv heads, the ranks of decays and gates, streams
and norm groups, the order of the layer types, chunks below and above a page or a key tile, filters of no, one and several
taps, routers that choose one, some or all experts, groups of one expert)."""
from __future__ import annotations

import functools
import json
from typing import Dict, List, Sequence, Tuple

import numpy as np
import torch

import helpers as H
import plain_notirax as pn
from ruvenex_cases import check_bf16


def _att(heads, kv, dim, vdim, scale, cap, chunk):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap, "mask": None if chunk is None else {"size": chunk}}


def _delta(heads, kv, dim, vdim, conv, ra, rg):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": ra, "gate_rank": rg}


def _moe(experts, top, ff, limit, scale, groups=None):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale,
                                      "groups": None if groups is None else {"count": groups[0], "keep": groups[1]}},
            "expert": {"ff": ff, "limit": limit}}


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def _base(vocab, width, eps, groups, streams, layers):
    return {"architecture": "Notirax", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "streams": streams, "layers": layers}


CASES: Dict[str, dict] = {
    # attention first, chunks of 24 (a page and a half), two value heads a key head, an attention layer without chunks
    "a": _base(200, 64, 1e-5, 4, 2, [
        _layer("attention", _att(4, 2, 16, 24, 0.3, 6.0, 24), _moe(6, 2, 24, 2.0, 1.5, (3, 2))),
        _layer("channel_delta", _delta(4, 2, 16, 32, 4, 8, 16), _moe(4, 1, 40, 3.0, 1.0)),
        _layer("attention", _att(4, 4, 16, 16, 0.25, 9.0, None), _moe(8, 3, 16, 1.0, 2.0, (2, 1)))]),
    # nothing a multiple of eight; six layers; five streams and three norm groups; chunks of 5 and 33; no cap; a layer
    # without feed-forward; groups of one expert each; a router that uses every expert; filters of no and of one tap
    "b": _base(97, 36, 3e-6, 3, 5, [
        _layer("channel_delta", _delta(3, 1, 10, 7, 3, 3, 5), None),
        _layer("attention", _att(3, 1, 10, 7, 0.4, None, 33), _moe(4, 4, 10, 1.5, 0.7, (4, 4))),
        _layer("attention", _att(2, 2, 6, 9, 0.5, 2.0, 5), _moe(9, 1, 5, 2.5, 3.0, (3, 1))),
        _layer("channel_delta", _delta(2, 2, 5, 11, 0, 2, 1), _moe(6, 2, 7, 0.8, 1.0, (6, 3))),
        _layer("channel_delta", _delta(4, 2, 6, 6, 1, 4, 4), None),
        _layer("attention", _att(1, 1, 12, 5, 0.3, 4.0, 17), _moe(5, 3, 9, 2.0, 1.2))]),
    # sizes the tensor-core kernels take: keys and values of 64 and 128 in both orders, chunks of 150 (across key tiles of
    # 128 and pages) and of 128, no chunks, six heads on two kv heads, twelve on four, states of 128 x 64; one norm group
    "c": _base(256, 128, 2e-6, 1, 4, [
        _layer("attention", _att(6, 2, 64, 64, 0.12, 8.0, 150), _moe(8, 2, 32, 2.0, 1.5, (4, 2))),
        _layer("channel_delta", _delta(3, 3, 24, 40, 2, 16, 8), _moe(4, 2, 64, 1.5, 1.0, (2, 1))),
        _layer("attention", _att(12, 4, 64, 128, 0.1, 12.0, None), None),
        _layer("attention", _att(2, 1, 128, 64, 0.09, None, 128), _moe(3, 2, 64, 7.0, 0.8)),
        _layer("channel_delta", _delta(2, 1, 128, 64, 3, 24, 32), _moe(16, 4, 16, 2.0, 2.5, (4, 2)))]),
    # one plain residual sum instead of streams
    "d": {k: v for k, v in _base(120, 48, 1e-6, 2, None, [
        _layer("channel_delta", _delta(2, 1, 16, 16, 3, 4, 6), _moe(4, 2, 16, 2.0, 1.0, (2, 2))),
        _layer("attention", _att(4, 1, 8, 12, 0.35, 5.0, 40), _moe(4, 2, 24, 2.0, 1.5))]).items() if k != "streams"},
}


def spec_of(cfg: dict):
    return H.spec_of(cfg)


CLUSTERS = 4


def make_weights(cfg: dict, seed: int, dtype=torch.bfloat16, sharp: float = 0.0, decisive: bool = False) -> Dict[str, torch.Tensor]:
    """Random weights; with ``sharp`` the queries' matrices of the attention layers are multiplied by it, so that attention
    weights are peaked: a position's result then hangs on single keys (the first of its chunk, a key hundreds of
    positions back), and a wrong key or a chunk one token off shows. With ``decisive`` (for bfloat16, where a close
    call may turn either way) tokens carry one of a few directions that the routers read, each router with well
    separated scores per direction."""
    from infer_b200.weights import random_weights
    W = random_weights(spec_of(cfg), seed, dtype)
    g = torch.Generator().manual_seed(seed)
    for i, l in enumerate(cfg["layers"]):
        if l["type"] == "attention":
            for n in ("q", "k", "v", "o"):                      # of a size that matters beside the other terms
                W[f"l{i}.mix.{n}"] = (W[f"l{i}.mix.{n}"].float() * 6.0).to(dtype)
            W[f"l{i}.mix.k.b"] = (W[f"l{i}.mix.k.b"].float() * 20.0).to(dtype)
            if sharp:
                W[f"l{i}.mix.q"] = (W[f"l{i}.mix.q"].float() * sharp).to(dtype)
    embed = W["embed"].float() * 25.0
    if decisive:
        U = torch.linalg.qr(torch.randn(cfg["width"], CLUSTERS, generator=g)).Q.T         # [CLUSTERS, width]
        embed += 3.0 * cfg["width"] ** 0.5 * U[torch.arange(cfg["vocab"]) % CLUSTERS]
        for i, l in enumerate(cfg["layers"]):
            if l.get("mlp"):
                W[f"l{i}.mlp.router"] = (_separated(l["mlp"]["router"], g) @ U * (1.5 / cfg["width"] ** 0.5)).to(dtype)
    W["embed"] = embed.to(dtype)
    return W


def _separated(router: dict, g: torch.Generator) -> torch.Tensor:
    """[experts, CLUSTERS] logits: per direction, random experts of random kept groups lie well above the rest of their
    groups, and those above the experts of the other groups."""
    E, top = router["experts"], router["top"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    count, keep = groups["count"], groups["keep"]
    per = E // count
    z = torch.full((CLUSTERS, E), -2.5)
    for c in range(CLUSTERS):
        kept = torch.randperm(count, generator=g)[:keep]
        members = torch.cat([torch.arange(per) + int(k) * per for k in kept])
        z[c, members] = -0.6
        order = torch.argsort(torch.rand(keep, per, generator=g), dim=1)                   # take turns among the kept groups
        picks = (order + (kept * per)[:, None]).T.reshape(-1)[:top]
        z[c, picks] = 1.3
    return (z + 0.2 * torch.rand(z.shape, generator=g)).T


def random_ids(cfg: dict, n: int, seed: int) -> List[int]:
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def plain_weights(cfg: dict, W: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    if cfg.get("streams"):
        return W
    W = dict(W)
    for i in range(len(cfg["layers"])):
        for q in ("hc1", "hc2"):
            W[f"l{i}.{q}.in"] = W[f"l{i}.{q}.out"] = torch.ones(1)
            W[f"l{i}.{q}.mix"] = torch.ones(1, 1)
    return W


@functools.lru_cache(maxsize=64)
def _oracle(cfg_json: str, seed: int, sharp: float, compute: str, ids: Tuple[int, ...], rounding: str):
    cfg = json.loads(cfg_json)
    W = plain_weights(cfg, H.as_compute(make_weights(cfg, seed, torch.bfloat16, sharp, compute == "bfloat16"), getattr(torch, compute)))
    if rounding == "none":
        return pn.forward(cfg, W, list(ids)).numpy()
    with pn.rounded(getattr(torch, rounding)):
        return pn.forward(cfg, W, list(ids)).numpy()


def oracle(cfg: dict, seed: int, compute: torch.dtype, ids: Sequence[int], rounding=None, sharp: float = 0.0) -> np.ndarray:
    n = lambda d: str(d).replace("torch.", "")
    return _oracle(json.dumps(cfg, sort_keys=True), seed, float(sharp), n(compute), tuple(int(i) for i in ids),
                   "none" if rounding is None else n(rounding))


CLOSE_CALL = 0.02      # a router's gap between its last chosen and first refused score below which bfloat16 roundings may turn the choice


@functools.lru_cache(maxsize=64)
def _router_gaps(cfg_json: str, seed: int, sharp: float, ids: Tuple[int, ...]) -> np.ndarray:
    cfg = json.loads(cfg_json)
    W = plain_weights(cfg, H.as_compute(make_weights(cfg, seed, torch.bfloat16, sharp, True), torch.bfloat16))
    gaps: List[torch.Tensor] = []
    pn.forward(cfg, W, list(ids), None, gaps)
    return torch.stack(gaps).min(dim=0).values.numpy() if gaps else np.full(len(ids), np.inf)


def check(cfg: dict, seed: int, dtype: torch.dtype, got: Dict[str, Dict[int, np.ndarray]], reqs: Dict[str, List[int]],
          sharp: float = 0.0, what: str = ""):
    """The engine's rows against the plain implementation. In bfloat16, positions from the first one at which a
    router's choice is a close call are left out (the other expert is as right an answer there, and every later
    position reads what that one left in the caches and states). The float32 comparison leaves out nothing and is
    the sharp one; cuttings are compared bit by bit there."""
    for rid, ids in reqs.items():
        ref = oracle(cfg, seed, dtype, ids, None, sharp)
        rows = sorted(got[rid])
        if dtype != torch.float32:
            gaps = _router_gaps(json.dumps(cfg, sort_keys=True), seed, float(sharp), tuple(int(i) for i in ids))
            close = np.nonzero(gaps < CLOSE_CALL)[0]
            upto = int(close[0]) if len(close) else len(ids)
            rows = [p for p in rows if p < upto]
            if not rows:
                continue
        g = np.stack([got[rid][p] for p in rows])
        if dtype == torch.float32:
            H.check_f32(g, ref[rows], f"{what}/{rid}")
        else:
            check_bf16(g, ref[rows], oracle(cfg, seed, dtype, ids, torch.bfloat16, sharp)[rows], f"{what}/{rid}", factor=4.0)
