"""Bolelix: typed configuration and its translation into a ModelSpec.

A decoder whose layers have one norm that both sublayers read, and a factor per channel on what each adds:

    n = rmsnorm(x);    x <- x + ls1 * mixer(n) + ls2 * feed_forward(n)                     (the last term absent without one)

(block kind "parallel_scaled", parts/block.py; the sum of a layer and the norm of the next are one kernel). The token
table's rows are multiplied by a constant; the same kind of norm precedes the output matrix. Three kinds of layer, in
any order:

"mamba2"     a state space layer with a matrix state per head that fades by one number per head and token, behind a short
             causal filter (parts/state_space.py)
"attention"  grouped-query softmax attention (parts/attention.py): channels i and i + dims / 2 of a head rotated with
             frequencies divided by a constant, every q and k head over its root mean square, a sliding window that keeps
             the first keys, one gate per head. A layer with ``kv_from: j`` has no keys and values of its own: it
             reads what layer j left in its cache (the run order names layer j's cache with write_cache False), with its
             own queries and mask
"mlstm"      matrix memory with exponential input gates, forget gates, a running maximum and a normaliser
             (parts/matrix_memory.py)

Feed-forward: a mixture of gated experts whose router takes the softmax over the chosen logits only
(parts/routed_ff.py), or none.

config.json keys (all sizes and constants come from there or from the tensors' shapes; tensor names are fixed):

    architecture "Bolelix"; vocab; width; norm.eps; embedding.scale; layers[i] = {type, mixer, mlp}
      type "mamba2":    mixer {heads, vdim, state, groups (= 1), conv (taps, = 1), norm_groups (= 1)}
      type "attention": mixer {heads, kv_heads (= heads), dim, vdim (= dim), scale, mask: {size, keep_first} | null,
                               rot: {base, dims, scaling: {factor} | null} | null, kv_from: layer index | absent}
      type "mlstm":     mixer {heads, dim, vdim (= dim), gate_cap}
      mlp {kind: "moe", router: {experts, top}, expert: {ff}} | null

Tensors: embed, final.norm, head, and per layer l<i>.: norm1, ls1, ls2, mix.* and mlp.* as the parts name them.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple, Union

from ..config.registry import Architecture, ConfigError, register_architecture
from ..config.specs import LayerCall, LayerSpec, ModelSpec, PartSpec

NAME = "Bolelix"
DEFAULT_MAX_POSITIONS = 1 << 20       # the design states no limit; an engine's own sequence limit sizes its tables
MEMORY_FLOOR = 1e-6                   # what the design adds to the matrix memory's denominator


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int
    factor: float = 1.0                # every frequency is divided by it


@dataclass(frozen=True)
class SoftmaxMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None
    keep_first: int = 0
    rot: Optional[Rotation] = None
    kv_from: Optional[int] = None


@dataclass(frozen=True)
class StateSpaceMixer:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int


@dataclass(frozen=True)
class MemoryMixer:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class RoutedFF:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class BolelixLayer:
    mixer: Union[SoftmaxMixer, StateSpaceMixer, MemoryMixer]
    mlp: Optional[RoutedFF]


@dataclass(frozen=True)
class BolelixConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: Tuple[BolelixLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS


def _get(raw, key: str, where: str):
    if not isinstance(raw, Mapping) or key not in raw:
        raise ConfigError(f"config.json: {where} is missing key {key!r}")
    return raw[key]


def _int(raw, key, where, minimum=1) -> int:
    v = _get(raw, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v < minimum:
        raise ConfigError(f"config.json: {where}.{key} must be an integer >= {minimum}, got {v!r}")
    return v


def _opt_int(raw, key, where, minimum=1) -> Optional[int]:
    return _int(raw, key, where, minimum) if isinstance(raw, Mapping) and raw.get(key) is not None else None


def _num(raw, key, where, positive=False) -> float:
    v = _get(raw, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or (positive and v <= 0):
        raise ConfigError(f"config.json: {where}.{key} must be a{' positive' if positive else ''} number, got {v!r}")
    return float(v)


def _multiple(a: int, b: int, what_a: str, what_b: str) -> None:
    if a % b:
        raise ConfigError(f"config.json: {what_a} ({a}) must be a multiple of {what_b} ({b})")


def _softmax_mixer(raw, where: str) -> SoftmaxMixer:
    heads = _int(raw, "heads", where)
    kv = _opt_int(raw, "kv_heads", where) or heads
    _multiple(heads, kv, f"{where}.heads", "kv_heads")
    dim = _int(raw, "dim", where)
    vdim = _opt_int(raw, "vdim", where) or dim
    mask, rot = raw.get("mask"), raw.get("rot")
    window = _int(mask, "size", where + ".mask") if mask is not None else None
    keep = (_opt_int(mask, "keep_first", where + ".mask", 0) or 0) if mask is not None else 0
    rotation = None
    if rot is not None:
        dims = _int(rot, "dims", where + ".rot", 2)
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim ({dim}), got {dims}")
        sc = rot.get("scaling")
        rotation = Rotation(_num(rot, "base", where + ".rot", positive=True), dims,
                            _num(sc, "factor", where + ".rot.scaling", positive=True) if sc is not None else 1.0)
    return SoftmaxMixer(heads, kv, dim, vdim, _num(raw, "scale", where), window, keep, rotation, _opt_int(raw, "kv_from", where, 0))


def _mixer(kind: str, raw, where: str):
    if kind == "attention":
        return _softmax_mixer(raw, where)
    heads = _int(raw, "heads", where)
    if kind == "mamba2":
        vdim, groups, norm_groups = _int(raw, "vdim", where), _opt_int(raw, "groups", where) or 1, _opt_int(raw, "norm_groups", where) or 1
        _multiple(heads, groups, f"{where}.heads", "groups")
        _multiple(heads * vdim, norm_groups, f"{where}: heads * vdim", "norm_groups")
        return StateSpaceMixer(heads, vdim, _int(raw, "state", where), groups, _opt_int(raw, "conv", where) or 1, norm_groups)
    dim = _int(raw, "dim", where)
    return MemoryMixer(heads, dim, _opt_int(raw, "vdim", where) or dim, _num(raw, "gate_cap", where, positive=True))


def _mlp(raw, where: str):
    if raw is None:
        return None
    kind = _get(raw, "kind", where)
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not a feed-forward of this design ('moe')")
    router, expert = _get(raw, "router", where), _get(raw, "expert", where)
    experts, top = _int(router, "experts", where + ".router"), _int(router, "top", where + ".router")
    if top > experts:
        raise ConfigError(f"config.json: {where}.router: {top} of {experts} experts cannot be chosen")
    return RoutedFF(experts, top, _int(expert, "ff", where + ".expert"))


def _check_shared(layers) -> None:
    for i, l in enumerate(layers):
        m = l.mixer
        if not isinstance(m, SoftmaxMixer) or m.kv_from is None:
            continue
        where = f"config.json: layers[{i}].mixer.kv_from"
        if m.kv_from >= i:
            raise ConfigError(f"{where} must name an earlier layer, got {m.kv_from}")
        owner = layers[m.kv_from].mixer
        if not isinstance(owner, SoftmaxMixer) or owner.kv_from is not None:
            raise ConfigError(f"{where}: layer {m.kv_from} has no keys and values of its own")
        if (m.kv_heads, m.dim, m.vdim, m.rot) != (owner.kv_heads, owner.dim, owner.vdim, owner.rot):
            raise ConfigError(f"{where}: kv_heads, dim, vdim and rotation of layer {m.kv_from} differ")


def parse(raw: Mapping[str, Any]) -> BolelixConfig:
    layers = _get(raw, "layers", "the configuration")
    if not isinstance(layers, (list, tuple)) or not layers:
        raise ConfigError("config.json: 'layers' must be a non-empty list")
    out = []
    for i, l in enumerate(layers):
        where = f"layers[{i}]"
        kind = _get(l, "type", where)
        if kind not in ("attention", "mamba2", "mlstm"):
            raise ConfigError(f"config.json: {where}.type {kind!r} is not a layer of this design ('attention', 'mamba2', 'mlstm')")
        out.append(BolelixLayer(_mixer(kind, _get(l, "mixer", where), where + ".mixer"), _mlp(l.get("mlp"), where + ".mlp")))
    _check_shared(out)
    max_positions = raw.get("max_positions", DEFAULT_MAX_POSITIONS)
    if isinstance(max_positions, bool) or not isinstance(max_positions, int) or max_positions <= 0:
        raise ConfigError(f"config.json: max_positions must be a positive integer, got {max_positions!r}")
    emb = raw.get("embedding")
    return BolelixConfig(vocab=_int(raw, "vocab", "the configuration"), width=_int(raw, "width", "the configuration"),
                         eps=_num(_get(raw, "norm", "the configuration"), "eps", "norm", positive=True),
                         embedding_scale=_num(emb, "scale", "embedding") if emb is not None and emb.get("scale") is not None else 1.0,
                         layers=tuple(out), max_positions=max_positions)


def _mixer_dict(m) -> Tuple[str, Dict[str, Any]]:
    if isinstance(m, StateSpaceMixer):
        return "mamba2", {"heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "conv": m.taps, "norm_groups": m.norm_groups}
    if isinstance(m, MemoryMixer):
        return "mlstm", {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap}
    d: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                         "mask": {"size": m.window, "keep_first": m.keep_first} if m.window is not None else None, "rot": None}
    if m.rot is not None:
        d["rot"] = {"base": m.rot.base, "dims": m.rot.dims, "scaling": {"factor": m.rot.factor}}
    if m.kv_from is not None:
        d["kv_from"] = m.kv_from
    return "attention", d


def to_dict(cfg: BolelixConfig) -> Dict[str, Any]:
    layers = []
    for l in cfg.layers:
        kind, mixer = _mixer_dict(l.mixer)
        f = l.mlp
        mlp = {"kind": "moe", "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.ff}} if f is not None else None
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    d = {"architecture": NAME, "vocab": cfg.vocab, "width": cfg.width, "norm": {"eps": cfg.eps},
         "embedding": {"scale": cfg.embedding_scale}, "layers": layers}
    if cfg.max_positions != DEFAULT_MAX_POSITIONS:
        d["max_positions"] = cfg.max_positions
    return d


def _cache_reach(layers, owner: int) -> Tuple[Optional[int], int]:
    """(window, kept first keys) of the pages that layer ``owner`` fills: what it and every layer that reads them see."""
    readers = [l.mixer for i, l in enumerate(layers) if isinstance(l.mixer, SoftmaxMixer) and (i == owner or l.mixer.kv_from == owner)]
    if any(m.window is None for m in readers):
        return None, 0
    return max(m.window for m in readers), max(m.keep_first for m in readers)


def _mixer_spec(cfg: BolelixConfig, i: int, prefix: str) -> PartSpec:
    m, W = cfg.layers[i].mixer, cfg.width
    if isinstance(m, StateSpaceMixer):
        return PartSpec("state_space", {"hidden_size": W, "num_heads": m.heads, "v_head_dim": m.vdim, "state_size": m.state,
                                        "groups": m.groups, "filter_taps": m.taps, "norm_groups": m.norm_groups, "norm_eps": cfg.eps,
                                        "names": {"in": "in", "filter": "conv", "filter_bias": "conv.b", "dt_bias": "dt_bias",
                                                  "a_log": "A_log", "skip": "D", "norm": "norm", "o": "o"}}, prefix)
    if isinstance(m, MemoryMixer):
        return PartSpec("matrix_memory", {"hidden_size": W, "num_heads": m.heads, "head_dim": m.dim, "v_head_dim": m.vdim,
                                          "gate_cap": m.gate_cap, "floor": MEMORY_FLOOR, "norm_eps": cfg.eps,
                                          "names": {"q": "q", "k": "k", "v": "v", "gate": "g", "o": "o", "norm": "norm", "input": "i",
                                                    "input_bias": "i.b", "forget": "f", "forget_bias": "f.b"}}, prefix)
    window, keep = _cache_reach(cfg.layers, m.kv_from if m.kv_from is not None else i)
    params: Dict[str, Any] = {
        "hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim,
        "window": m.window, "keep_first": m.keep_first if m.window is not None else 0, "cache_window": window, "cache_keep_first": keep,
        "softmax_scale": m.scale, "position": None, "qk_unit_norm_eps": cfg.eps, "head_gate": True, "own_kv": m.kv_from is None,
        "names": {"q": "q", "k": "k", "v": "v", "o": "o", "gate": "g"}}
    if m.rot is not None:
        params["position"] = PartSpec("rotary_interpolated", {"theta": m.rot.base, "rotary_dims": m.rot.dims, "head_dim": m.dim,
                                                              "layout": "half", "linear_factor": m.rot.factor,
                                                              "max_positions": cfg.max_positions})
    return PartSpec("attention", params, prefix)


def _norm(W: int, eps: float, name: str, prefix: str) -> PartSpec:
    return PartSpec("rmsnorm", {"size": W, "eps": eps, "weight_name": name}, prefix)


def to_spec(cfg: BolelixConfig) -> ModelSpec:
    W = cfg.width
    layers, schedule, optional, cache_of = [], [], [], {}
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        scale = lambda name: ("connection", PartSpec("channel_scale", {"size": W, "weight_name": name}, p))
        parts = {"norm": ("norm", _norm(W, cfg.eps, "norm1", p)), "mixer": ("mixer", _mixer_spec(cfg, i, p + "mix.")),
                 "mixer_scale": scale("ls1")}
        if l.mlp is not None:
            parts["feed_forward"] = ("feed_forward", PartSpec(
                "routed_experts", {"hidden_size": W, "experts": l.mlp.experts, "top": l.mlp.top, "expert_size": l.mlp.ff,
                                   "router_kind": "softmax_top", "expert_kind": "swish_glu"}, p + "mlp."))
            parts["feed_forward_scale"] = scale("ls2")
        else:
            optional.append(p + "ls2")                   # a factor on nothing may be stored all the same
        layers.append(LayerSpec("parallel_scaled", parts))
        kv_from = getattr(l.mixer, "kv_from", None)
        owner = i if kv_from is None else kv_from
        if kv_from is None:
            cache_of[i] = len(cache_of)
        schedule.append(LayerCall(i, cache_of[owner], kv_from is None))
    spec = ModelSpec(
        architecture=NAME, hidden_size=W, vocab_size=cfg.vocab, max_positions=cfg.max_positions, layers=tuple(layers),
        schedule=tuple(schedule), final_norm=_norm(W, cfg.eps, "final.norm", ""),
        embedding=PartSpec("token_table", {"vocab_size": cfg.vocab, "hidden_size": W, "weight_name": "embed",
                                           "scale": cfg.embedding_scale}, ""),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": W, "tied": False, "weight_name": "head"}, ""),
        eos_token_id=None, optional_tensors=tuple(optional), stream=PartSpec("pending_sum", {"size": W}))
    spec.validate()
    return spec


ARCHITECTURE = register_architecture(Architecture(NAME, parse, to_spec, to_dict))
