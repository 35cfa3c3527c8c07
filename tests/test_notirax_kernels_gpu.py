"""The kernels behind Notirax's parts, each alone against the plain implementation's function for the same mechanism
(float64), in float and bfloat16 storage, over segments of unequal length with state carried between steps."""
import math

import numpy as np
import pytest
import torch

import plain_notirax as pn
from infer_b200 import ops
from test_fozerax_kernels_gpu import _paged
from test_ruvenex_kernels_gpu import _Step

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F = torch.float64


def _tol(dtype):
    return dict(rtol=2e-2, atol=2e-2) if dtype == torch.bfloat16 else dict(rtol=2e-5, atol=2e-5)


# ----------------------------------------------------------------------------------------------- the streams

@pytest.mark.parametrize("n,width,groups", [(1, 36, 3), (2, 30, 1), (3, 96, 4), (4, 1536, 8), (4, 1000, 2), (5, 48, 6), (7, 72, 12), (11, 40, 10),
                                            (2, 13000, 4), (6, 27, 27)])
def test_streams_take_in_a_result_and_give_the_next_normalised_rows(n, width, groups):
    g = torch.Generator().manual_seed(n * width)
    T, eps = 5, 1e-4
    rnd = lambda *s: torch.randn(*s, generator=g)
    x, y, M, b, a, w = 3 * rnd(T, n, width), rnd(T, width), rnd(n, n), rnd(n), rnd(n), rnd(width)
    d = lambda t: t.to(DEV)
    X = pn.write_streams(x.double(), M, b, y.double())
    want = pn.grouped_norm(pn.read_streams(X, a), w, eps, groups)
    xd = d(x)
    out_x, normed = ops.stream_link(xd, n, torch.float32, d(y), d(M), d(b), d(a), d(w), eps, groups)
    assert out_x.data_ptr() == xd.data_ptr()                                   # rewritten in place
    assert torch.allclose(out_x.double().cpu(), X, rtol=2e-5, atol=5e-5)
    assert torch.allclose(normed.double().cpu(), want, rtol=2e-5, atol=5e-5)
    # the compute-dtype rows are the float rows rounded
    _, half = ops.stream_link(d(x), n, torch.bfloat16, d(y), d(M), d(b), d(a), d(w), eps, groups)
    assert torch.equal(half.cpu(), normed.cpu().to(torch.bfloat16))
    # nothing pending: the streams stay
    same, normed = ops.stream_link(xd, n, torch.float32, in_w=d(a), norm_w=d(w), eps=eps, groups=groups)
    assert same is xd and torch.allclose(normed.double().cpu(), pn.grouped_norm(pn.read_streams(X, a), w, eps, groups), rtol=2e-5, atol=5e-5)
    # one row stands for all streams; a result makes them differ, in a buffer of their own
    row = rnd(T, width)
    rd = d(row)
    all_equal = row[:, None, :].repeat(1, n, 1).double()
    _, normed = ops.stream_link(rd, n, torch.float32, in_w=d(a), norm_w=d(w), eps=eps, groups=groups)
    assert torch.allclose(normed.double().cpu(), pn.grouped_norm(pn.read_streams(all_equal, a), w, eps, groups), rtol=1e-4, atol=1e-4)
    got, _ = ops.stream_link(rd, n, torch.float32, d(y), d(M), d(b), d(a), d(w), eps, groups)
    assert torch.allclose(got.double().cpu().view(T, n, width), pn.write_streams(all_equal, M, b, y.double()), rtol=2e-5, atol=5e-5)
    # the end: the plain sum of picked rows, what is pending included, nothing stored
    xd = d(x)
    rows = torch.tensor([3, 0, 3], dtype=torch.int32, device=DEV)
    kept, normed = ops.stream_link(xd, n, torch.float32, d(y), d(M), d(b), None, d(w), eps, groups, rows=rows)
    assert torch.equal(kept.cpu(), x)
    assert torch.allclose(normed.double().cpu(), pn.grouped_norm(X.sum(dim=1), w, eps, groups)[[3, 0, 3]], rtol=2e-5, atol=5e-5)
    _, total = ops.stream_link(xd, n, torch.float32, d(y), d(M), d(b), store=False)
    assert torch.allclose(total.double().cpu(), X.sum(dim=1), rtol=2e-5, atol=1e-4)


def test_a_stream_row_does_not_depend_on_its_neighbours():
    g = torch.Generator().manual_seed(3)
    n, W = 3, 192
    x, y = torch.randn(9, n, W, generator=g).to(DEV), torch.randn(9, W, generator=g).to(DEV)
    M, b, a, w = (torch.randn(*s, generator=g).to(DEV) for s in ((n, n), (n,), (n,), (W,)))
    X, N = ops.stream_link(x.clone(), n, torch.float32, y, M, b, a, w, 1e-5, 4)
    for t in (0, 8):
        X1, N1 = ops.stream_link(x[t:t + 1].clone(), n, torch.float32, y[t:t + 1].contiguous(), M, b, a, w, 1e-5, 4)
        assert torch.equal(X1[0], X[t]) and torch.equal(N1[0], N[t])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("width", [8, 37, 256])
def test_table_rows_with_sinusoidal_positions(width, dtype):
    g = torch.Generator().manual_seed(width)
    V = 50
    table = torch.randn(V, width, generator=g).to(dtype)
    pos = torch.tensor([0, 1, 2, 17, 4095, 65537, 1000003], dtype=torch.int32)
    ids = torch.tensor([3, 49, 0, 7, 7, 12, -1], dtype=torch.int32)
    freq = pn.POSITION_BASE ** (-2.0 * torch.arange((width + 1) // 2, dtype=F) / width)
    step = _Step([7], [0], [1])
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    feedback = torch.tensor([5, 21], dtype=torch.int32, device=DEV)             # the id -1 stands for the slot's last token
    out = ops.embedding_sinusoid(table.to(DEV), ids.to(DEV), pos.to(DEV), freq.to(DEV), status, feedback, step.token_seg, step.seg_slot, 1.5)
    ids[-1] = 21
    want = 1.5 * table.double()[ids.long()] + pn.sinusoid(pos, width)
    assert torch.allclose(out.double().cpu(), want, rtol=1e-6, atol=1e-6) and int(status.item()) == 0
    ids[2] = V                                                                  # outside the table: zeros and the status word
    out = ops.embedding_sinusoid(table.to(DEV), ids.to(DEV), pos.to(DEV), freq.to(DEV), status)
    assert int(status.item()) == 1 and float(out[2].abs().sum()) == 0.0


# ----------------------------------------------------------------------------------------------- attention

def _case(H, G, d, dv, n, dtype, seed):
    g = torch.Generator().manual_seed(seed)
    q, k, v = (torch.randn(n, h, s, generator=g).to(dtype).double() for h, s in ((H, d), (G, d), (G, dv)))
    talk = torch.eye(H) + 0.4 * torch.randn(H, H, generator=g)
    return q, k, v, talk, g


def _stand_out(q, k, key, query, head):
    """One key's score from one query and head becomes large."""
    if 0 <= key <= query:
        d, r = q.shape[2], q.shape[1] // k.shape[1]
        k[key, head // r] += 3.0 * q[query, head] / q[query, head].norm() * math.sqrt(d)


def _rows(q, k, v, at, dtype, col0, pad=0):
    """Packed rows [col0 columns | q | k | v | pad] of the tokens ``at``."""
    n = len(at)
    parts = [torch.full((n, col0), 9.0, dtype=F), q[at].reshape(n, -1), k[at].reshape(n, -1), v[at].reshape(n, -1), torch.full((n, pad), 9.0, dtype=F)]
    return torch.cat(parts, dim=1).to(dtype).to(DEV).contiguous()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("chunk,cap,with_talk", [(None, 4.0, True), (5, 0.0, True), (64, 3.0, False), (70, 2.0, True), (130, 30.0, True), (256, 0.0, False)])
@pytest.mark.parametrize("sizes", [(6, 2, 64, 48), (3, 3, 10, 7), (8, 1, 32, 64), (28, 4, 96, 128), (12, 2, 128, 128)])
def test_capped_exchanged_scores_in_chunks_plain_and_split(sizes, chunk, cap, with_talk, dtype):
    """Single tokens around borders of chunks, pages (16) and key tiles (64), and the first positions, beside a longer
    segment. For each, the first key of its chunk stands out, and the last key of the chunk before, and key 0."""
    H, G, d, dv = sizes
    n, scale = 300, 0.15
    q, k, v, talk, g = _case(H, G, d, dv, n, dtype, d + (chunk or 0))
    if not with_talk:
        talk = None
    c = chunk or n
    probes = sorted({p for p in (0, 1, 15, 16, 17, 63, 64, 65, 127, 128, 200, 299, c - 1, c, c + 1, 2 * c - 1, 2 * c, 2 * c + 3) if p < n})
    for i, p in enumerate(probes):
        _stand_out(q, k, p // c * c, p, i % H)
        _stand_out(q, k, p // c * c - 1, p, (i + 1) % H)
        _stand_out(q, k, 0, p, (i + 2) % H)
    k = k.to(dtype).double()
    want = pn.attend(q, k, v, scale, cap, talk, pn.visible(n, chunk))
    row = list(np.random.default_rng(1).permutation(24))[:19]
    kc, vc = _paged([k], [v], [row], 24, G, d, dv, dtype)
    kc, vc = kc.to(DEV), vc.to(DEV)
    S = len(probes) + 1
    table = torch.tensor([row] * S, dtype=torch.int32, device=DEV)
    step = _Step([1] * len(probes) + [37], probes + [180], list(range(S)))
    step.seg_lens, step.max_q_len, step.max_ctx_len = step.lens, 37, n
    at = probes + list(range(180, 217))
    rows = _rows(q, k, v, at, dtype, 8, 3 if d == 10 else 8)
    td = talk.to(DEV).contiguous() if talk is not None else None
    args = (rows, 8, kc, vc, table, step, H, G, d, dv, None, chunk, scale, cap, td)
    plain = ops.talk_attention(*args).double().cpu().view(-1, H, dv)
    assert torch.allclose(plain, want[at], **_tol(dtype))
    assert int(step.status.item()) == 0
    out = torch.full((len(at), H * dv), 7.0, dtype=dtype, device=DEV)
    got = ops.talk_attention_split(*args, out=out, single_only=True)
    if dtype == torch.float32 or d % 32 or dv % 8:
        assert got is None
        return
    got = got.double().cpu().view(-1, H, dv)
    assert torch.allclose(got[:len(probes)], want[probes], **_tol(dtype))
    assert float((got[len(probes):] - 7.0).abs().sum()) == 0.0                 # the longer segment's rows were left alone
    # tokens whose own keys and values are still in their rows, each the last of its request: stored by the same kernel
    for p in (probes[-1], probes[3]):
        page, place = row[p // 16], p % 16
        kp, vp = kc.clone(), vc.clone()
        kp[page, :, place:], vp[page, :, place:] = float("nan"), float("nan")
        one = _Step([1], [p], [0])
        one.seg_lens, one.max_q_len, one.max_ctx_len = [1], 1, p + 1
        o = ops.talk_attention_split(_rows(q, k, v, [p], dtype, 8, 8), 8, kp, vp, table[:1].contiguous(), one, H, G, d, dv, None, chunk, scale, cap, td,
                                     fresh_cols=(8 + H * d, 8 + (H + G) * d))
        assert torch.equal(kp[page, :, place], kc[page, :, place]) and torch.equal(vp[page, :, place], vc[page, :, place])
        assert bool(torch.isnan(kp[page, :, place + 1:].float()).all()) and int(one.status.item()) == 0
        assert torch.equal(o.double().cpu().view(H, dv), got[probes.index(p)])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("sizes", [(3, 10, 7), (2, 64, 128)])
def test_keys_and_values_go_to_their_pages(sizes, dtype):
    G, d, dv = sizes
    lens, pos0 = [21, 1, 6], [13, 40, 0]
    step = _Step(lens, pos0, [0, 1, 2])
    T = sum(lens)
    rows = torch.randn(T, 8 + G * (d + dv) + 8, generator=torch.Generator().manual_seed(d)).to(dtype).to(DEV)
    table = torch.tensor([[3, 7, 1, -1], [5, 0, 2, 9], [4, -1, -1, -1]], dtype=torch.int32, device=DEV)
    kc = torch.full((12, G, 16, d), float("nan"), dtype=dtype, device=DEV)
    vc = torch.full((12, G, 16, dv), float("nan"), dtype=dtype, device=DEV)
    ops.kv_store(rows, 8, 8 + G * d, step, table, kc, vc, G, d, dv)
    seg, pos = step.token_seg.cpu().tolist(), step.positions.cpu().tolist()
    for t in range(T):
        page, place = int(table[seg[t], pos[t] // 16]), pos[t] % 16
        assert torch.equal(kc[page, :, place].reshape(-1), rows[t, 8:8 + G * d])
        assert torch.equal(vc[page, :, place].reshape(-1), rows[t, 8 + G * d:8 + G * (d + dv)])
    assert int(torch.isnan(kc.float()).sum()) == (12 * 16 - T) * G * d and int(step.status.item()) == 0


@pytest.mark.parametrize("chunk,cap,with_talk", [(None, 5.0, True), (128, 2.0, True), (150, 0.0, True), (40, 3.0, True), (333, 30.0, False)])
@pytest.mark.parametrize("sizes", [(6, 2, 64, 64), (12, 2, 128, 128), (4, 4, 64, 128), (5, 1, 128, 64), (28, 4, 128, 128), (1, 1, 64, 64)])
def test_prompt_portions_on_the_tensor_cores(sizes, chunk, cap, with_talk):
    """A portion of 470 tokens behind 30 cached ones (four query tiles, the last ragged), one of 2 tokens, and a single
    token of a third request, in one step. Keys at the two sides of chunk borders stand out for rows around them."""
    from infer_b200 import fast_ops
    H, G, d, dv = sizes
    scale, dtype = 0.11, torch.bfloat16
    lengths, first = (500, 90, 161), (30, 89, 159)
    cases = [_case(H, G, d, dv, n, dtype, 7 * i + d + (chunk or 0)) for i, n in enumerate(lengths)]
    talk = cases[0][3] if with_talk else None
    c = chunk or 500
    q, k = cases[0][0], cases[0][1]
    for i, p in enumerate((31, 127, 128, 300, 499, c - 1, c, c + 1, 2 * c, 3 * c - 1)):
        if p < 500:
            for m, key in enumerate((p // c * c, p // c * c - 1, 0)):
                _stand_out(q, k, key, p, (i + m) % H)
    seqs = [(cs[0], cs[1].to(dtype).double(), cs[2]) for cs in cases]
    want = [pn.attend(*sq, scale, cap, talk, pn.visible(n, chunk)) for sq, n in zip(seqs, lengths)]
    tables = [list(range(3, 35)), [40, 36, 38, 37, 41, 39], [50, 44, 53, 45, 52, 46, 51, 47, 49, 48, 54]]
    kc, vc = _paged([s[1] for s in seqs], [s[2] for s in seqs], tables, 56, G, d, dv, dtype)
    table = torch.full((3, 40), -1, dtype=torch.int32)
    for i, t in enumerate(tables):
        table[i, :len(t)] = torch.tensor(t, dtype=torch.int32)
        if chunk is not None:                                  # pages of chunks that have passed have been given back
            table[i, :first[i] // chunk * chunk // 16] = -1
    step = _Step([n - f for n, f in zip(lengths, first)], list(first), [0, 1, 2])
    step.seg_lens, step.seg_pos0 = step.lens, torch.tensor(step.pos0, dtype=torch.int32, device=DEV)
    step.max_q_len, step.max_ctx_len = 470, 500
    rows = torch.cat([_rows(*s, list(range(f, n)), dtype, 8, 8) for s, f, n in zip(seqs, first, lengths)]).contiguous()
    td = talk.to(DEV).contiguous() if talk is not None else None
    args = (rows, 8, kc.to(DEV), vc.to(DEV), table.to(DEV), step, H, G, d, dv, None, chunk, scale, cap, td)
    fast_ops.device_state(torch.device(DEV)).status.zero_()
    out = fast_ops.talk_attention_prefill(*args)
    assert out is not None
    assert ops.talk_attention_split(*args, out=out, single_only=True) is out
    assert int(fast_ops.device_state(torch.device(DEV)).status.item()) == 0 and int(step.status.item()) == 0
    got = out.double().cpu().view(-1, H, dv)
    ref = torch.cat([w[f:] for w, f in zip(want, first)])
    assert torch.allclose(got, ref, rtol=3e-2, atol=4e-2), float((got - ref).abs().max())
    assert float((got - ref).pow(2).mean().sqrt()) < 6e-3
    # with little room for scores the query tiles go in rounds: the same bits
    limit = fast_ops.TALK_SCORES_MAX_BYTES
    try:
        fast_ops.TALK_SCORES_MAX_BYTES = 1
        again = fast_ops.talk_attention_prefill(*args)
    finally:
        fast_ops.TALK_SCORES_MAX_BYTES = limit
    assert torch.equal(again[:470], out[:470]) and torch.equal(again[471:], out[471:])


# ----------------------------------------------------------------------------------------------- the delta rule

# a key size below, at and above each number of state rows a lane keeps; value sizes that are no multiple of four
SCAN_SIZES = [(2, 1, 16, 32), (3, 3, 5, 9), (2, 2, 64, 64), (4, 2, 40, 20), (2, 1, 128, 64), (1, 1, 160, 128), (3, 1, 33, 3), (2, 2, 64, 130)]


def _delta_case(H, G, d, dv, taps, n, seed):
    g = torch.Generator().manual_seed(seed)
    C = 2 * G * d + H * dv
    return {"u": torch.randn(n, C, generator=g), "b": torch.randn(n, H, generator=g), "z": 2 * torch.randn(n, H * d, generator=g)}


def _delta_reference(x, w, a_log, dt_bias, H, G, d, dv):
    n, r = x["u"].shape[0], H // G
    u = pn.silu(pn.causal_filter(x["u"].double(), w.T) if w is not None else x["u"].double())
    q, k, v = u[:, :G * d].view(n, G, d), u[:, G * d:2 * G * d].view(n, G, d), u[:, 2 * G * d:].view(n, H, dv)
    q, k = pn.unit(q) * d ** -0.5, pn.unit(k)
    g = pn.channel_decays(x["z"].double(), a_log, dt_bias, H)
    beta = torch.sigmoid(x["b"].double())
    return torch.stack([pn.channel_delta_scan(q[:, h // r], k[:, h // r], v[:, h], g[:, h], beta[:, h])[0] for h in range(H)], dim=1)


@pytest.mark.parametrize("taps", [0, 1, 2, 4])
@pytest.mark.parametrize("sizes", SCAN_SIZES)
def test_delta_rule_with_decays_per_channel_over_steps(sizes, taps):
    """Preparation and scan over two requests of unequal length in one step after the other (portions down to one token),
    then one request over other cuttings: the same bits."""
    H, G, d, dv = sizes
    g = torch.Generator().manual_seed(sum(sizes))
    C = 2 * G * d + H * dv
    a_log, dt_bias = torch.log(0.1 + 2 * torch.rand(H, generator=g)), torch.randn(H * d, generator=g) - 1.0
    w = torch.randn(taps, C, generator=g) if taps else None                    # tap-major
    seqs = {0: _delta_case(H, G, d, dv, taps, 45, 1), 2: _delta_case(H, G, d, dv, taps, 23, 2)}
    ref = {s: _delta_reference(x, w, a_log, dt_bias, H, G, d, dv) for s, x in seqs.items()}
    dec_col, sc_col = ops.delta_columns(H, G, d, dv, True)
    dev = lambda t: None if t is None else t.to(DEV).contiguous()

    def run(parts, lens, at, slots, S, tails, inline):
        step = _Step(lens, at, slots)
        rows = torch.cat([torch.cat([torch.full((m, 4), 9.0), x["u"][a:a + m], x["b"][a:a + m]], dim=1) for x, a, m in zip(parts, at, lens)])
        logits = torch.cat([torch.cat([torch.full((m, 3), 9.0), x["z"][a:a + m]], dim=1) for x, a, m in zip(parts, at, lens)])
        prep = ops.delta_prepare(dev(rows), 4, 0, 4 + C, dev(w), tails, dev(a_log), dev(dt_bias), pn.UNIT_EPS, d ** -0.5, step, H, G, d, dv,
                                 inline, dev(logits), 3)
        if tails is not None and not inline:
            ops.tail_update(dev(rows), 4, tails, step.seg_start, step.seg_slot)
        return ops.state_scan(ops.SCAN_CHANNEL_DELTA, prep, 0, G * d, 2 * G * d, prep, dec_col, S, step.seg_start, step.seg_slot, H, H // G, d, dv,
                              True, max(lens), scalar_col=sc_col).cpu()

    def fresh():
        S = torch.full((3, H, d, dv), float("nan"), device=DEV)
        tails = torch.full((3, taps - 1, C), float("nan"), device=DEV) if taps > 1 else None
        for t in (S, tails):
            if t is not None:
                t[0].zero_(), t[2].zero_()
        return S, tails
    S, tails = fresh()
    at, got = {0: 0, 2: 0}, {0: [], 2: []}
    for lens in ([1, 2], [2, 1], [17, 3], [1, 1], [24, 16]):
        o = run([seqs[0], seqs[2]], lens, [at[0], at[2]], [0, 2], S, tails, taps > 1 and max(lens) == 1)
        for s, m, a in ((0, lens[0], 0), (2, lens[1], lens[0])):
            got[s].append(o[a:a + m])
            at[s] += m
    for s in (0, 2):
        assert torch.allclose(torch.cat(got[s]).double().view(-1, H, dv), ref[s], rtol=5e-5, atol=5e-5)
    assert bool(torch.isnan(S[1]).all())
    for cuts in ([45], [1] * 45, [2] * 22 + [1]):
        S1, t1 = fresh()
        a, outs = 0, []
        for m in cuts:
            outs.append(run([seqs[0]], [m], [a], [0], S1, t1, taps > 1 and m == 1))
            a += m
        assert torch.equal(torch.cat(outs), torch.cat(got[0])) and torch.equal(S1[0], S[0])


# ----------------------------------------------------------------------------------------------- the router

@pytest.mark.parametrize("E,top,count,keep", [(20, 3, 2, 1), (8, 8, 1, 1), (12, 3, 4, 2), (6, 2, 6, 3), (40, 6, 5, 5), (64, 4, 8, 3), (1, 1, 1, 1)])
def test_router_with_sigmoid_scores_and_groups_of_two_best(E, top, count, keep):
    g = torch.Generator().manual_seed(E + top)
    logits = 2.0 * torch.randn(65, E, generator=g)
    router = {"experts": E, "top": top, "scale": 1.7, "groups": {"count": count, "keep": keep}}
    chosen, w = pn.route(logits.double(), router)
    want = torch.zeros(65, E, dtype=F).scatter_(1, chosen, w)
    weights, got = ops.route(logits.to(DEV), top, count, keep, want_chosen=True, sigmoid=True, group_best=2, renormalise=False, mult=1.7)
    assert torch.allclose(weights.double().cpu(), want, rtol=1e-5, atol=1e-6)
    assert torch.equal(got.cpu().long(), chosen)
