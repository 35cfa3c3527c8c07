"""Notirax: typed configuration and its translation into a ModelSpec.

A pre-norm decoder over several residual streams (parts/streams.py, block kind "hyper_prenorm"). The token table's rows
plus a sinusoidal position vector (parts/vocab.py) fill n equal streams; a sublayer f reads one combination of them and
writes into all of them:

    u = sum_s a_s x_s;   y = f(norm(u));   x_t <- sum_s M[s, t] x_s + b_t y

The norms divide each of `norm.groups` equal parts of a row by the part's own root mean square (parts/rmsnorm.py). The
streams' sum passes the final norm; the logits are its products with the token table. Two kinds of layer, in any order:

"attention"      grouped-query softmax attention without positions in its scores (parts/attention.py): biased projections,
                 scores capped by a hyperbolic tangent and then exchanged among the heads through a learned matrix, keys
                 of the query's own chunk of positions only
"channel_delta"  the gated delta rule with a decay per head and key channel behind short causal filters, decays and
                 output gate through low ranks (parts/delta_rule.py)

Feed-forward: a mixture of clipped gated experts, a sigmoid router with groups whose score is the sum of a group's two
best, weights as they are times a constant (parts/routed_ff.py); or none.

config.json keys (all sizes and constants come from there or from the tensors' shapes; tensor names are fixed):

    architecture "Notirax"; vocab; width; norm {eps, groups (= 1)}; streams (absent: one plain residual sum);
    layers[i] = {type, mixer, mlp}
      type "attention":     mixer {heads, kv_heads (= heads), dim, vdim (= dim), scale, softcap | null, mask: {size} | null}
      type "channel_delta": mixer {heads, kv_heads (= heads), dim, vdim (= dim), conv (0: no filter)}
      mlp {kind: "moe", router: {experts, top, scale (= 1), groups: {count, keep} | null}, expert: {ff, limit}} | null

A configuration written for a random model also carries ``decay_rank`` and ``gate_rank`` (channel_delta), which a
checkpoint's tensors otherwise state.

Tensors: embed, final.norm, and per layer l<i>.: norm1, norm2, hc1.*, hc2.*, mix.* and mlp.* as the parts name them.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple, Union

from ..config.registry import Architecture, ConfigError, register_architecture
from ..config.specs import LayerCall, LayerSpec, ModelSpec, PartSpec

NAME = "Notirax"
DEFAULT_MAX_POSITIONS = 1 << 20       # the design states no limit; an engine's own sequence limit sizes its tables
# constants that the design fixes
POSITION_BASE = 10000.0               # of the sinusoidal position vector
UNIT_EPS = 1e-6                       # inside the root when q and k of the delta rule are made unit vectors
EXPERT_SLOPE = 1.702                  # an expert's g * sigmoid(slope * g)


@dataclass(frozen=True)
class TalkingMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float]
    chunk: Optional[int]


@dataclass(frozen=True)
class ChannelDeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: Optional[int]          # None: the stored tensors state it
    gate_rank: Optional[int]


@dataclass(frozen=True)
class RoutedFF:
    experts: int
    top: int
    scale: float
    groups: int
    keep: int
    ff: int
    limit: float


@dataclass(frozen=True)
class NotiraxLayer:
    mixer: Union[TalkingMixer, ChannelDeltaMixer]
    mlp: Optional[RoutedFF]


@dataclass(frozen=True)
class NotiraxConfig:
    vocab: int
    width: int
    eps: float
    norm_groups: int
    streams: Optional[int]
    layers: Tuple[NotiraxLayer, ...]
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


def _mixer(kind: str, raw, where: str):
    heads = _int(raw, "heads", where)
    kv = _opt_int(raw, "kv_heads", where) or heads
    if heads % kv:
        raise ConfigError(f"config.json: {where}.heads ({heads}) must be a multiple of kv_heads ({kv})")
    dim = _int(raw, "dim", where)
    vdim = _opt_int(raw, "vdim", where) or dim
    if kind == "channel_delta":
        return ChannelDeltaMixer(heads, kv, dim, vdim, _opt_int(raw, "conv", where, 0) or 0, _opt_int(raw, "decay_rank", where),
                                 _opt_int(raw, "gate_rank", where))
    mask = raw.get("mask")
    return TalkingMixer(heads, kv, dim, vdim, _num(raw, "scale", where),
                        _num(raw, "softcap", where, positive=True) if raw.get("softcap") is not None else None,
                        _int(mask, "size", where + ".mask") if mask is not None else None)


def _mlp(raw, where: str) -> Optional[RoutedFF]:
    if raw is None:
        return None
    kind = _get(raw, "kind", where)
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not a feed-forward of this design ('moe')")
    router, expert = _get(raw, "router", where), _get(raw, "expert", where)
    rw = where + ".router"
    experts, top = _int(router, "experts", rw), _int(router, "top", rw)
    groups = router.get("groups")
    count = _int(groups, "count", rw + ".groups") if groups is not None else 1
    keep = _int(groups, "keep", rw + ".groups") if groups is not None else 1
    if experts % count or keep > count or top > keep * (experts // count):
        raise ConfigError(f"config.json: {rw}: {experts} experts in {count} groups of which {keep} are kept "
                          f"cannot give {top} experts a token")
    return RoutedFF(experts, top, _num(router, "scale", rw) if router.get("scale") is not None else 1.0, count, keep,
                    _int(expert, "ff", where + ".expert"), _num(expert, "limit", where + ".expert", positive=True))


def parse(raw: Mapping[str, Any]) -> NotiraxConfig:
    layers = _get(raw, "layers", "the configuration")
    if not isinstance(layers, (list, tuple)) or not layers:
        raise ConfigError("config.json: 'layers' must be a non-empty list")
    out = []
    for i, l in enumerate(layers):
        where = f"layers[{i}]"
        kind = _get(l, "type", where)
        if kind not in ("attention", "channel_delta"):
            raise ConfigError(f"config.json: {where}.type {kind!r} is not a layer of this design ('attention', 'channel_delta')")
        out.append(NotiraxLayer(_mixer(kind, _get(l, "mixer", where), where + ".mixer"), _mlp(l.get("mlp"), where + ".mlp")))
    max_positions = raw.get("max_positions", DEFAULT_MAX_POSITIONS)
    if isinstance(max_positions, bool) or not isinstance(max_positions, int) or max_positions <= 0:
        raise ConfigError(f"config.json: max_positions must be a positive integer, got {max_positions!r}")
    norm = _get(raw, "norm", "the configuration")
    width, groups = _int(raw, "width", "the configuration"), _opt_int(norm, "groups", "norm") or 1
    if width % groups:
        raise ConfigError(f"config.json: width ({width}) must be a multiple of norm.groups ({groups})")
    return NotiraxConfig(vocab=_int(raw, "vocab", "the configuration"), width=width, eps=_num(norm, "eps", "norm", positive=True),
                         norm_groups=groups, streams=_opt_int(raw, "streams", "the configuration"), layers=tuple(out),
                         max_positions=max_positions)


def to_dict(cfg: NotiraxConfig) -> Dict[str, Any]:
    layers = []
    for l in cfg.layers:
        m = l.mixer
        mixer: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim}
        if isinstance(m, TalkingMixer):
            kind = "attention"
            mixer.update(scale=m.scale, softcap=m.softcap, mask={"size": m.chunk} if m.chunk is not None else None)
        else:
            kind = "channel_delta"
            mixer["conv"] = m.taps
            for key, rank in (("decay_rank", m.decay_rank), ("gate_rank", m.gate_rank)):
                if rank is not None:
                    mixer[key] = rank
        f = l.mlp
        mlp = None if f is None else {"kind": "moe", "router": {"experts": f.experts, "top": f.top, "scale": f.scale,
                                                                "groups": {"count": f.groups, "keep": f.keep}},
                                      "expert": {"ff": f.ff, "limit": f.limit}}
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    d = {"architecture": NAME, "vocab": cfg.vocab, "width": cfg.width, "norm": {"eps": cfg.eps, "groups": cfg.norm_groups}, "layers": layers}
    if cfg.streams is not None:
        d["streams"] = cfg.streams
    if cfg.max_positions != DEFAULT_MAX_POSITIONS:
        d["max_positions"] = cfg.max_positions
    return d


def _mixer_spec(m, W: int, eps: float, prefix: str) -> PartSpec:
    if isinstance(m, TalkingMixer):
        return PartSpec("attention", {
            "hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim, "qkv_bias": True,
            "o_bias": True, "softmax_scale": m.scale, "position": None, "score_cap": m.softcap, "head_exchange": True, "chunk": m.chunk,
            "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "o_bias": "o.b",
                      "talk": "talk"}}, prefix)
    return PartSpec("channel_delta_rule", {
        "hidden_size": W, "num_heads": m.heads, "num_qk_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim, "filter_taps": m.taps,
        "norm_eps": eps, "unit_eps": UNIT_EPS, "decay_rank": m.decay_rank, "gate_rank": m.gate_rank,
        "names": {"q": "q", "k": "k", "v": "v", "q_filter": "q.conv", "k_filter": "k.conv", "v_filter": "v.conv", "beta": "b",
                  "a_log": "A_log", "dt_bias": "dt_bias", "decay_low": "a1", "decay_up": "a2", "gate_low": "g1", "gate_up": "g2",
                  "norm": "norm", "o": "o"}}, prefix)


def to_spec(cfg: NotiraxConfig) -> ModelSpec:
    W = cfg.width
    norm = lambda name, prefix: PartSpec("rmsnorm", {"size": W, "eps": cfg.eps, "groups": cfg.norm_groups, "weight_name": name}, prefix)
    layers, optional = [], []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        link = lambda q: {} if cfg.streams is None else {q[0]: ("connection", PartSpec("hyper", {"streams": cfg.streams}, p + q[1]))}
        parts = {"mixer_norm": ("norm", norm("norm1", p)), **link(("mixer_link", "hc1.")),
                 "mixer": ("mixer", _mixer_spec(l.mixer, W, cfg.eps, p + "mix."))}
        if l.mlp is not None:
            f = l.mlp
            parts.update({"feed_forward_norm": ("norm", norm("norm2", p)), **link(("feed_forward_link", "hc2.")),
                          "feed_forward": ("feed_forward", PartSpec("routed_experts", {
                              "hidden_size": W, "experts": f.experts, "top": f.top, "groups": f.groups, "keep": f.keep, "expert_size": f.ff,
                              "limit": f.limit, "slope": EXPERT_SLOPE, "router_kind": "sigmoid_groups", "out_scale": f.scale}, p + "mlp."))})
        else:                                            # what belongs to a sublayer that is not there may be stored all the same
            optional += [p + "norm2"] + [p + "hc2." + n for n in ("in", "out", "mix")]
        layers.append(LayerSpec("prenorm" if cfg.streams is None else "hyper_prenorm", parts))
    spec = ModelSpec(
        architecture=NAME, hidden_size=W, vocab_size=cfg.vocab, max_positions=cfg.max_positions, layers=tuple(layers),
        schedule=tuple(LayerCall(i, i) for i in range(len(layers))),
        final_norm=norm("final.norm", ""),
        embedding=PartSpec("token_table", {"vocab_size": cfg.vocab, "hidden_size": W, "weight_name": "embed", "sinusoid_base": POSITION_BASE}, ""),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": W, "tied": True}, ""),
        eos_token_id=None, optional_tensors=tuple(optional),
        stream=None if cfg.streams is None else PartSpec("copies", {"streams": cfg.streams}, ""))
    spec.validate()
    return spec


ARCHITECTURE = register_architecture(Architecture(NAME, parse, to_spec, to_dict))
