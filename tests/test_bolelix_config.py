"""Bolelix without a GPU: configuration, tensor names, cache needs with pages that several layers read, and the plain
implementation's own consistency."""
import copy
import math

import pytest
import torch

import bolelix_cases as BC
import helpers as H
import infer_b200.models  # noqa: F401  (registers the architectures)
import infer_b200.parts  # noqa: F401
import plain_bolelix as pb
from infer_b200.cache.manager import CacheManager
from infer_b200.config import parse_config
from infer_b200.config.registry import ConfigError
from infer_b200.models import load_preset
from infer_b200.parts.base import PagedKVNeed, StateNeed, part_class
from infer_b200.weights.binder import WeightsError, check_weights, expected_tensors

F = torch.float64


@pytest.mark.parametrize("name", sorted(BC.CASES))
def test_config_round_trip_and_tensor_names(name):
    cfg = BC.CASES[name]
    arch, typed = parse_config(cfg)
    assert arch.name == "Bolelix"
    assert arch.parse(arch.to_dict(typed)) == typed
    names = expected_tensors(arch.to_spec(typed))
    W = cfg["width"]
    assert names["embed"][0] == names["head"][0] == (cfg["vocab"], W) and names["final.norm"][0] == (W,)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H_, dv = m["heads"], m["vdim"]
        assert names[p + "norm1"][0] == names[p + "ls1"][0] == (W,) and ((p + "ls2") in names) == (l["mlp"] is not None)
        assert (p + "norm2") not in names and names[p + "mix.o"][0] == (W, H_ * dv)
        if l["type"] == "attention":
            assert names[p + "mix.q"][0] == (H_ * m["dim"], W) and names[p + "mix.g"][0] == (H_, W)
            assert ((p + "mix.k") in names) == ((p + "mix.v") in names) == (m.get("kv_from") is None)
            if m.get("kv_from") is None:
                assert names[p + "mix.k"][0] == (m["kv_heads"] * m["dim"], W) and names[p + "mix.v"][0] == (m["kv_heads"] * dv, W)
        elif l["type"] == "mamba2":
            ch = H_ * dv + 2 * m["groups"] * m["state"]
            assert names[p + "mix.in"][0] == (H_ * dv + ch + H_, W) and names[p + "mix.conv"][0] == (ch, m["conv"])
            assert names[p + "mix.conv.b"][0] == (ch,) and names[p + "mix.norm"][0] == (H_ * dv,)
            assert {names[p + "mix." + n][0] for n in ("dt_bias", "A_log", "D")} == {(H_,)}
        else:
            assert names[p + "mix.q"][0] == names[p + "mix.k"][0] == (H_ * m["dim"], W)
            assert names[p + "mix.v"][0] == names[p + "mix.g"][0] == (H_ * dv, W) and names[p + "mix.norm"][0] == (H_ * dv,)
            assert names[p + "mix.i"][0] == names[p + "mix.f"][0] == (H_, W) and names[p + "mix.i.b"][0] == names[p + "mix.f.b"][0] == (H_,)
        if l["mlp"]:
            E, ff = l["mlp"]["router"]["experts"], l["mlp"]["expert"]["ff"]
            assert names[p + "mlp.router"][0] == (E, W) and names[p + f"mlp.e{E - 1}.gate"][0] == (ff, W)
            assert names[p + f"mlp.e{E - 1}.down"][0] == (W, ff) and (p + f"mlp.e{E}.up") not in names


def test_presets_parse():
    for n in ("tiny-bolelix", "bolelix-1.5b", "bolelix-7b"):
        arch, typed = parse_config(load_preset(n))
        assert arch.name == "Bolelix" and arch.to_spec(typed).layers


def _broken(path, value=None, delete=False):
    cfg = copy.deepcopy(BC.CASES["a"])
    node = cfg
    for k in path[:-1]:
        node = node[k]
    if delete:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    return cfg


@pytest.mark.parametrize("path,value,delete,word", [
    (("norm",), None, True, "norm"),
    (("norm", "eps"), 0, False, "eps"),
    (("layers", 0, "type"), "gla", False, "not a layer"),
    (("layers", 0, "mixer", "groups"), 3, False, "groups"),
    (("layers", 0, "mixer", "norm_groups"), 5, False, "norm_groups"),
    (("layers", 0, "mixer", "state"), None, True, "state"),
    (("layers", 1, "mixer", "kv_heads"), 3, False, "multiple"),
    (("layers", 1, "mixer", "scale"), None, True, "scale"),
    (("layers", 1, "mixer", "mask", "size"), 0, False, "size"),
    (("layers", 1, "mixer", "mask", "keep_first"), -1, False, "keep_first"),
    (("layers", 1, "mixer", "rot", "dims"), 18, False, "dims"),
    (("layers", 1, "mixer", "rot", "scaling", "factor"), 0, False, "factor"),
    (("layers", 2, "mixer", "kv_from"), 0, False, "no keys and values"),
    (("layers", 2, "mixer", "kv_from"), 4, False, "earlier"),
    (("layers", 4, "mixer", "kv_from"), 2, False, "no keys and values"),
    (("layers", 2, "mixer", "rot", "base"), 999.0, False, "differ"),
    (("layers", 3, "mixer", "gate_cap"), None, True, "gate_cap"),
    (("layers", 0, "mlp", "router", "top"), 7, False, "cannot be chosen"),
    (("layers", 0, "mlp", "kind"), "dense", False, "not a feed-forward"),
])
def test_refusals_name_the_key(path, value, delete, word):
    with pytest.raises(ConfigError) as e:
        parse_config(_broken(path, value, delete))
    assert word in str(e.value)


def test_options_that_may_be_absent():
    cfg = copy.deepcopy(BC.CASES["a"])
    for k in ("groups", "conv", "norm_groups"):
        del cfg["layers"][0]["mixer"][k]
    cfg["layers"] = cfg["layers"][:2] + cfg["layers"][3:4]
    m = cfg["layers"][1]["mixer"]
    m["mask"] = None
    for k in ("kv_heads", "vdim", "rot"):
        del m[k]
    del cfg["layers"][2]["mixer"]["vdim"], cfg["embedding"]
    arch, typed = parse_config(cfg)
    s, a, x = (l.mixer for l in typed.layers)
    assert (s.groups, s.taps, s.norm_groups) == (1, 1, 1) and (a.kv_heads, a.vdim, a.window, a.keep_first, a.rot) == (4, 16, None, 0, None)
    assert x.vdim == x.dim == 16 and typed.embedding_scale == 1.0
    spec = arch.to_spec(typed)
    assert spec.stream.kind == "pending_sum" and spec.layers[1].part("mixer")["position"] is None


def test_one_error_lists_what_is_missing():
    cfg = BC.CASES["a"]
    W = BC.make_weights(cfg, 3)
    spec = BC.spec_of(cfg)
    check_weights(W, spec)
    broken = dict(W)
    del broken["l3.mix.f.b"], broken["l2.ls1"]
    broken["l0.mix.A_log"], broken["l2.mix.k"] = torch.zeros(3), torch.zeros(32, 64)     # a reader's keys are another layer's
    with pytest.raises(WeightsError) as e:
        check_weights(broken, spec)
    for word in ("l3.mix.f.b", "l2.ls1", "l0.mix.A_log", "l2.mix.k"):
        assert word in str(e.value)
    check_weights({**W, "l4.ls2": torch.ones(64)}, spec)                                 # a factor on nothing may be stored


# ----------------------------------------------------------------------------- the cache

class _NoDevice:
    """Enough of a runtime to build a part for its cache need (nothing is loaded)."""
    dtype = torch.float32
    device = torch.device("cpu")
    max_seq_len = 64

    def fast(self, op):
        return False


def _needs(cfg):
    spec = BC.spec_of(cfg)
    return spec, [part_class("mixer", ls.part("mixer").kind)(ls.part("mixer"), _NoDevice()).cache_need() for ls in spec.layers]


def test_layers_that_read_a_cache_need_what_its_writer_keeps():
    spec, needs = _needs(BC.CASES["a"])
    assert needs[1] == needs[2] == needs[4] == PagedKVNeed(2, 16, 40, keep_first=11)     # the widest window, the most kept keys
    assert [(c.cache, c.write_cache) for c in spec.schedule] == [(0, True), (1, True), (1, False), (2, True), (1, False)]
    assert isinstance(needs[0], StateNeed) and needs[0].shapes["S"][0] == (4, 24, 16) and needs[0].shapes["tails"][0] == (3, 4 * 16 + 2 * 2 * 24)
    assert {k: v[0] for k, v in needs[3].shapes.items()} == {"S": (3, 16, 24), "n": (3, 16), "m": (3,)}
    spec, needs = _needs(BC.CASES["b"])
    assert needs[1] == needs[4] == PagedKVNeed(1, 10, None, 7)            # a reader without a mask: every position stays
    assert needs[3] == PagedKVNeed(2, 6, 5, 9) and "tails" not in needs[5].shapes          # a filter of one tap keeps nothing
    _, needs = _needs(BC.CASES["c"])
    assert needs[0] == needs[2] == PagedKVNeed(2, 64, 150, keep_first=140)


def test_pages_behind_the_widest_window_go_back_and_the_kept_ones_stay():
    spec, needs = _needs(BC.CASES["a"])
    mgr = CacheManager({c.cache: needs[c.layer] for c in spec.schedule if c.write_cache}, n_pages=12, page_size=16, n_slots=2)
    held = lambda: [p >= 0 for p in mgr.block_table("x", mgr.group_of_cache[1][0])]
    mgr.admit("x")
    assert mgr.reserve("x", 71)
    mgr.advance("x", 71)
    assert held() == [True, False, True, True, True]         # the next query (71) still reads key 32 of page 2; page 0 is kept
    mgr.reserve("x", 17)
    mgr.advance("x", 17)                                      # 88 positions: the window begins at 49, in page 3
    assert held() == [True, False, False, True, True, True]
    mgr.check_invariants()
    mgr.release("x")
    assert mgr.pages_in_use() == [0]


# ----------------------------------------------------------------------------- the plain implementation against itself

def test_what_a_window_with_kept_keys_sees():
    ok = pb.visible(6, 2, 1)
    assert [r.nonzero()[:, 0].tolist() for r in ok] == [[0], [0, 1], [0, 1, 2], [0, 2, 3], [0, 3, 4], [0, 4, 5]]


def test_rotation_turns_halves_and_keeps_lengths():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=F)
    rot = {"base": 16.0, "dims": 4, "scaling": {"factor": 2.0}}
    y = pb.rotate_halves(x, torch.tensor([3]), rot)[0, 0]
    a0, a1 = 3 / 2.0, 3 * 16.0 ** (-2 / 4) / 2.0
    want = [math.cos(a0) - 3 * math.sin(a0), 2 * math.cos(a1) - 4 * math.sin(a1), 3 * math.cos(a0) + math.sin(a0),
            4 * math.cos(a1) + 2 * math.sin(a1), 5.0]
    assert torch.allclose(y, torch.tensor(want, dtype=F)) and torch.allclose(y.norm(), x.norm())


def test_the_product_s_rotation_tables():
    from infer_b200.config.specs import PartSpec
    rt = _NoDevice()
    rot = part_class("position", "rotary_interpolated")(PartSpec("rotary_interpolated", {
        "theta": 500.0, "rotary_dims": 6, "head_dim": 9, "layout": "half", "linear_factor": 2.5, "max_positions": 64}), rt)
    cos, sin = rot.rotary_tables(40)
    a = torch.arange(40, dtype=F)[:, None] * pb.frequencies(6, 500.0, 2.5)[None, :]
    assert torch.allclose(cos.double(), torch.cos(a), atol=1e-7) and torch.allclose(sin.double(), torch.sin(a), atol=1e-7)


def test_scans_can_be_cut_anywhere_and_read_their_own_write():
    g = torch.Generator().manual_seed(0)
    q, k = (torch.randn(9, 5, generator=g, dtype=F) for _ in range(2))
    v, gg, dt = torch.randn(9, 7, generator=g, dtype=F), torch.rand(9, generator=g, dtype=F), torch.rand(9, generator=g, dtype=F)
    whole, S = pb.fading_scan(q, k, v, gg, dt, 0.7)
    x, Sx = pb.fading_scan(q[:4], k[:4], v[:4], gg[:4], dt[:4], 0.7)
    y, Sy = pb.fading_scan(q[4:], k[4:], v[4:], gg[4:], dt[4:], 0.7, Sx)
    assert torch.allclose(torch.cat([x, y]), whole) and torch.allclose(S, Sy)
    assert torch.allclose(whole[0], dt[0] * (k[0] * q[0]).sum() * v[0] + 0.7 * v[0])
    i, f = pb.memory_gates(4 * torch.randn(9, generator=g, dtype=F), torch.randn(9, generator=g, dtype=F), 3.0)
    assert float(i.abs().max()) < 3.0 and float(f.max()) < 0.0
    whole, S, n, m = pb.memory_scan(q, k, v, i, f)
    x, Sx, nx, mx = pb.memory_scan(q[:4], k[:4], v[:4], i[:4], f[:4])
    y, Sy, ny, my = pb.memory_scan(q[4:], k[4:], v[4:], i[4:], f[4:], Sx, nx, mx)
    assert torch.allclose(torch.cat([x, y]), whole) and torch.allclose(S, Sy) and torch.allclose(n, ny) and m == my


def test_the_running_maximum_starts_at_zero_and_only_rescales():
    """Without a maximum, S = sum of e^(i + later f) k v^T and the lower bound of the denominator is 1: the recurrence with
    its maximum is the same function (up to the constant that is added to the denominator)."""
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(6, d, generator=g, dtype=F) for d in (4, 4, 3))
    i, f = torch.randn(6, generator=g, dtype=F) * 2, -torch.rand(6, generator=g, dtype=F)
    S, n, want = torch.zeros(4, 3, dtype=F), torch.zeros(4, dtype=F), []
    for t in range(6):
        S = torch.exp(f[t]) * S + torch.exp(i[t]) * k[t][:, None] * v[t]
        n = torch.exp(f[t]) * n + torch.exp(i[t]) * k[t]
        want.append(S.T @ q[t] / max(abs(float(n @ q[t])), 1.0))
    assert torch.allclose(pb.memory_scan(q, k, v, i, f)[0], torch.stack(want), rtol=1e-4)


def test_softplus_and_the_router():
    z = torch.tensor([-800.0, -1.0, 0.0, 3.0, 800.0], dtype=F)
    assert torch.allclose(pb.softplus(z)[1:4], torch.log1p(torch.exp(z[1:4]))) and pb.softplus(z)[0] == 0 and pb.softplus(z)[4] == 800
    assert torch.allclose(pb.log_sigmoid(z)[1:4], torch.log(torch.sigmoid(z[1:4]))) and pb.log_sigmoid(z)[0] == -800
    chosen, w, gap = pb.route_top(torch.tensor([[0.0, 2.0, -1.0, 1.0]], dtype=F), 2)
    assert chosen.tolist() == [[1, 3]] and float(gap) == 1.0
    assert torch.allclose(w, torch.softmax(torch.tensor([[2.0, 1.0]], dtype=F), dim=-1))


@pytest.mark.parametrize("name", ["a", "b"])
def test_a_prefix_does_not_depend_on_what_follows(name):
    cfg = BC.CASES[name]
    Wc = H.as_compute(BC.make_weights(cfg, 5), torch.float32)
    ids = BC.random_ids(cfg, 50, 9)
    assert torch.allclose(pb.forward(cfg, Wc, ids)[:30], pb.forward(cfg, Wc, ids[:30]), atol=1e-12)
