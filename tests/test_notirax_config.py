"""Notirax without a GPU: configuration, tensor names, sizes that only a checkpoint states, cache needs with pages that
chunks give back, and the plain implementation's own consistency."""
import copy
import math

import pytest
import torch

import helpers as H
import infer_b200.models  # noqa: F401  (registers the architectures)
import infer_b200.parts  # noqa: F401
import notirax_cases as NC
import plain_notirax as pn
from infer_b200.cache.manager import CacheManager
from infer_b200.config import parse_config
from infer_b200.config.registry import ConfigError
from infer_b200.models import load_preset
from infer_b200.parts.base import PagedKVNeed, StateNeed, part_class
from infer_b200.weights.binder import WeightsError, check_weights, expected_tensors

F = torch.float64


@pytest.mark.parametrize("name", sorted(NC.CASES))
def test_config_round_trip_and_tensor_names(name):
    cfg = NC.CASES[name]
    arch, typed = parse_config(cfg)
    assert arch.name == "Notirax"
    assert arch.parse(arch.to_dict(typed)) == typed
    names = expected_tensors(arch.to_spec(typed))
    W, n = cfg["width"], cfg.get("streams")
    assert names["embed"][0] == (cfg["vocab"], W) and names["final.norm"][0] == (W,) and "head" not in names
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        hd, kd, hv, kv = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"], m["kv_heads"] * m["vdim"]
        assert names[p + "norm1"][0] == (W,) and ((p + "norm2") in names) == (l["mlp"] is not None)
        for q, there in (("hc1", True), ("hc2", l["mlp"] is not None)):
            assert ((p + q + ".mix") in names) == (there and n is not None)
        if n is not None:
            assert names[p + "hc1.in"][0] == names[p + "hc1.out"][0] == (n,) and names[p + "hc1.mix"][0] == (n, n)
        assert names[p + "mix.q"][0] == ((hd if l["type"] == "attention" else kd), W) and names[p + "mix.k"][0] == (kd, W)
        assert names[p + "mix.o"][0] == (W, hv)
        if l["type"] == "attention":
            assert names[p + "mix.v"][0] == (kv, W) and names[p + "mix.talk"][0] == (m["heads"], m["heads"])
            assert [names[p + f"mix.{x}.b"][0] for x in "qkvo"] == [(hd,), (kd,), (kv,), (W,)]
        else:
            ra, rg = m["decay_rank"], m["gate_rank"]
            assert names[p + "mix.v"][0] == (hv, W) and names[p + "mix.b"][0] == (m["heads"], W) and names[p + "mix.A_log"][0] == (m["heads"],)
            assert names[p + "mix.a1"][0] == (ra, W) and names[p + "mix.a2"][0] == (hd, ra) and names[p + "mix.dt_bias"][0] == (hd,)
            assert names[p + "mix.g1"][0] == (rg, W) and names[p + "mix.g2"][0] == (hv, rg) and names[p + "mix.norm"][0] == (m["vdim"],)
            assert ((p + "mix.q.conv") in names) == (m["conv"] > 0)
            if m["conv"]:
                assert names[p + "mix.k.conv"][0] == (kd, m["conv"]) and names[p + "mix.v.conv"][0] == (hv, m["conv"])
        if l["mlp"]:
            E, ff = l["mlp"]["router"]["experts"], l["mlp"]["expert"]["ff"]
            assert names[p + "mlp.router"][0] == (E, W) and names[p + f"mlp.e{E - 1}.gate"][0] == (ff, W)
            assert names[p + f"mlp.e{E - 1}.down"][0] == (W, ff) and (p + f"mlp.e{E}.up") not in names


def test_presets_parse():
    for n in ("tiny-notirax", "notirax-1.5b", "notirax-7b"):
        arch, typed = parse_config(load_preset(n))
        assert arch.name == "Notirax" and arch.to_spec(typed).layers


def _broken(path, value=None, delete=False):
    cfg = copy.deepcopy(NC.CASES["a"])
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
    (("norm", "groups"), 5, False, "groups"),
    (("norm", "eps"), 0, False, "eps"),
    (("streams",), 0, False, "streams"),
    (("layers", 0, "type"), "gla", False, "not a layer"),
    (("layers", 0, "mixer", "kv_heads"), 3, False, "multiple"),
    (("layers", 0, "mixer", "scale"), None, True, "scale"),
    (("layers", 0, "mixer", "softcap"), -1.0, False, "softcap"),
    (("layers", 0, "mixer", "mask", "size"), 0, False, "size"),
    (("layers", 1, "mixer", "conv"), -1, False, "conv"),
    (("layers", 1, "mixer", "dim"), None, True, "dim"),
    (("layers", 2, "mlp", "router", "groups", "count"), 3, False, "cannot give"),
    (("layers", 2, "mlp", "router", "top"), 5, False, "cannot give"),
    (("layers", 0, "mlp", "expert", "limit"), 0, False, "limit"),
    (("layers", 0, "mlp", "kind"), "dense", False, "not a feed-forward"),
])
def test_refusals_name_the_key(path, value, delete, word):
    with pytest.raises(ConfigError) as e:
        parse_config(_broken(path, value, delete))
    assert word in str(e.value)


def test_options_that_may_be_absent():
    cfg = copy.deepcopy(NC.CASES["a"])
    m = cfg["layers"][0]["mixer"]
    m["mask"] = None
    for k in ("kv_heads", "vdim", "softcap"):
        del m[k]
    del cfg["norm"]["groups"], cfg["layers"][0]["mlp"]["router"]["groups"], cfg["layers"][0]["mlp"]["router"]["scale"], cfg["streams"]
    arch, typed = parse_config(cfg)
    t = typed.layers[0].mixer
    assert (t.kv_heads, t.vdim, t.softcap, t.chunk) == (4, 16, None, None) and typed.norm_groups == 1 and typed.streams is None
    f = typed.layers[0].mlp
    assert (f.groups, f.keep, f.scale) == (1, 1, 1.0)
    spec = arch.to_spec(typed)
    assert spec.stream is None and spec.layers[0].block == "prenorm" and spec.layers[0].part("mixer")["score_cap"] is None


def test_one_error_lists_what_is_missing_and_missing_ranks_are_read_from_the_tensors():
    cfg = copy.deepcopy(NC.CASES["a"])
    W = NC.make_weights(cfg, 3)
    del cfg["layers"][1]["mixer"]["decay_rank"], cfg["layers"][1]["mixer"]["gate_rank"]
    arch, typed = parse_config(cfg)
    spec = arch.to_spec(typed)
    check_weights(W, spec)
    broken = dict(W)
    del broken["l0.mix.talk"], broken["l2.hc2.mix"]
    broken["l1.mix.A_log"] = torch.zeros(3)
    with pytest.raises(WeightsError) as e:
        check_weights(broken, spec)
    for word in ("l0.mix.talk", "l2.hc2.mix", "l1.mix.A_log"):
        assert word in str(e.value)


def test_a_layer_without_feed_forward_may_have_its_tensors_stored_all_the_same():
    cfg = NC.CASES["b"]
    spec = NC.spec_of(cfg)
    W = NC.make_weights(cfg, 3)
    W.update({"l0.norm2": torch.ones(36), "l0.hc2.in": torch.ones(5), "l0.hc2.out": torch.ones(5), "l0.hc2.mix": torch.eye(5)})
    check_weights(W, spec)


# ----------------------------------------------------------------------------- the cache

class _NoDevice:
    """Enough of a runtime to build a part for its cache need (nothing is loaded)."""
    dtype = torch.float32
    device = torch.device("cpu")
    max_seq_len = 64

    def fast(self, op):
        return False


def test_cache_needs_and_pages_of_chunks_that_have_passed():
    spec = NC.spec_of(NC.CASES["b"])
    needs = {}
    for i, ls in enumerate(spec.layers):
        ps = ls.part("mixer")
        needs[i] = part_class("mixer", ps.kind)(ps, _NoDevice()).cache_need()
    assert isinstance(needs[0], StateNeed) and needs[0].shapes["S"][0] == (3, 10, 7) and needs[0].shapes["tails"][0] == (2, 2 * 10 + 3 * 7)
    assert needs[1] == PagedKVNeed(1, 10, None, 7, chunk=33) and needs[2] == PagedKVNeed(2, 6, None, 9, chunk=5)
    assert "tails" not in needs[3].shapes and "tails" not in needs[4].shapes           # filters of no and of one tap keep nothing
    mgr = CacheManager(needs, n_pages=12, page_size=16, n_slots=2)
    held = lambda cid: [p >= 0 for p in mgr.block_table("x", mgr.group_of_cache[cid][0])]
    mgr.admit("x")
    assert mgr.reserve("x", 32)
    mgr.advance("x", 32)
    assert held(1) == [True, True]                      # positions 0..31 lie in the chunk that the next query (32) still reads
    assert held(2) == [False, True]                     # chunks of 5: the next query reads from position 30
    assert mgr.reserve("x", 1)
    mgr.advance("x", 1)
    assert held(1) == [False, False, True]              # position 33 begins a chunk of 33: its page is 2
    assert mgr.reserve("x", 35)
    mgr.advance("x", 35)                                # 68 positions: the next query's chunk begins at 66, in page 4
    assert held(1) == [False] * 4 + [True]
    mgr.check_invariants()
    mgr.release("x")
    assert mgr.pages_in_use() == [0] * len(mgr.groups)
    mgr.admit("y")
    assert mgr.reserve("y", 40)                         # the pages that came back are used again
    mgr.check_invariants()


def test_needs_that_differ_in_their_chunk_form_groups_of_their_own():
    mgr = CacheManager({0: PagedKVNeed(2, 8, chunk=16), 1: PagedKVNeed(2, 8), 2: PagedKVNeed(2, 8, chunk=16), 3: PagedKVNeed(2, 8, chunk=24)},
                       n_pages=8, page_size=16, n_slots=1)
    assert len(mgr.groups) == 3 and mgr.group_of_cache[0][0] == mgr.group_of_cache[2][0]


# ----------------------------------------------------------------------------- the plain implementation against itself

def test_what_a_chunk_sees():
    ok = pn.visible(7, 3)
    assert [r.nonzero()[:, 0].tolist() for r in ok] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]
    assert pn.visible(4, None).tolist() == torch.tril(torch.ones(4, 4, dtype=torch.bool)).tolist()


def test_streams_read_and_write_as_stated():
    X = torch.tensor([[[1.0, 2.0], [3.0, 5.0]]], dtype=F)
    M, b, y = torch.tensor([[1.0, 10.0], [100.0, 1000.0]]), torch.tensor([2.0, 3.0]), torch.tensor([[0.5, 0.25]], dtype=F)
    out = pn.write_streams(X, M, b, y)                  # M is [from, to]
    assert out[0, 0].tolist() == [1 + 300 + 1.0, 2 + 500 + 0.5] and out[0, 1].tolist() == [10 + 3000 + 1.5, 20 + 5000 + 0.75]
    assert pn.read_streams(X, torch.tensor([1.0, -1.0])).tolist() == [[-2.0, -3.0]]


def test_norm_over_groups_and_positions():
    x = torch.tensor([[3.0, 4.0, 30.0, 40.0]], dtype=F)
    w = torch.tensor([1.0, 1.0, 1.0, 2.0])
    r = math.sqrt(12.5)
    assert torch.allclose(pn.grouped_norm(x, w, 0.0, 2), torch.tensor([[3 / r, 4 / r, 3 / r, 8 / r]], dtype=F))
    s = pn.sinusoid(torch.tensor([0, 3]), 5)
    assert s[0].tolist() == [0.0, 1.0, 0.0, 1.0, 0.0]
    f = 10000.0 ** (-2 / 5)
    assert torch.allclose(s[1], torch.tensor([math.sin(3), math.cos(3), math.sin(3 * f), math.cos(3 * f), math.sin(3 * f * f)], dtype=F))


def test_heads_exchange_capped_scores_before_the_softmax():
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(4, h, 3, generator=g, dtype=F) for h in (2, 1, 1))
    swap = torch.tensor([[0.0, 1.0], [1.0, 0.0]])
    seen = pn.visible(4, None)
    a, b = pn.attend(q, k, v, 0.5, 2.0, swap, seen), pn.attend(q, k, v, 0.5, 2.0, None, seen)
    assert torch.allclose(a[:, 0], b[:, 1]) and torch.allclose(a[:, 1], b[:, 0])
    assert abs(float(pn.softcap(torch.tensor(1e9, dtype=F), 2.0)) - 2.0) < 1e-12 and float(pn.softcap(torch.tensor(7.0), None)) == 7.0


def test_the_delta_scan_can_be_cut_anywhere_and_reads_its_own_write():
    g = torch.Generator().manual_seed(0)
    q, k, a = (torch.rand(9, 5, generator=g, dtype=F) for _ in range(3))
    v, beta = torch.randn(9, 7, generator=g, dtype=F), torch.rand(9, generator=g, dtype=F)
    whole, S = pn.channel_delta_scan(q, k, v, a, beta)
    x, Sx = pn.channel_delta_scan(q[:4], k[:4], v[:4], a[:4], beta[:4])
    y, Sy = pn.channel_delta_scan(q[4:], k[4:], v[4:], a[4:], beta[4:], Sx)
    assert torch.allclose(torch.cat([x, y]), whole) and torch.allclose(S, Sy)
    assert torch.allclose(whole[0], beta[0] * (k[0] * q[0]).sum() * v[0])       # an empty state: the current write alone
    assert torch.allclose(pn.channel_delta_scan(q, k, v, torch.zeros_like(a), beta)[0], beta[:, None] * (k * q).sum(-1, keepdim=True) * v)


def test_the_router_sums_a_groups_two_best_scores():
    z = torch.logit(torch.tensor([[0.9, 0.1, 0.2, 0.6, 0.55, 0.3]], dtype=F))
    assert torch.allclose(pn.group_scores(torch.sigmoid(z), 2), torch.tensor([[1.1, 1.15]], dtype=F))
    chosen, w = pn.route(z, {"top": 2, "scale": 2.0, "groups": {"count": 2, "keep": 1}})
    assert chosen.tolist() == [[3, 4]] and torch.allclose(w, torch.tensor([[1.2, 1.1]], dtype=F))
    chosen, w = pn.route(z, {"top": 1, "groups": {"count": 6, "keep": 2}})              # groups of one expert
    assert chosen.tolist() == [[0]] and torch.allclose(w, torch.tensor([[0.9]], dtype=F))


@pytest.mark.parametrize("name", ["b", "d"])
def test_a_prefix_does_not_depend_on_what_follows(name):
    cfg = NC.CASES[name]
    Wc = NC.plain_weights(cfg, H.as_compute(NC.make_weights(cfg, 5), torch.float32))
    ids = NC.random_ids(cfg, 50, 9)
    assert torch.allclose(pn.forward(cfg, Wc, ids)[:30], pn.forward(cfg, Wc, ids[:30]), atol=1e-12)
