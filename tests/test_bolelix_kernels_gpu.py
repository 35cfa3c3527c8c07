"""The kernels behind Bolelix's parts, each alone against the plain implementation's function for the same mechanism
(float64), in float and bfloat16 storage, over segments of unequal length with state carried between steps."""
import math

import numpy as np
import pytest
import torch

import plain_bolelix as pb
from infer_b200 import ops
from test_fozerax_kernels_gpu import _paged
from test_ruvenex_kernels_gpu import _Step

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F = torch.float64


def _tol(dtype):
    return dict(rtol=2e-2, atol=2e-2) if dtype == torch.bfloat16 else dict(rtol=2e-5, atol=2e-5)


# ----------------------------------------------------------------------------------------------- sum and norm

@pytest.mark.parametrize("width", [36, 27, 192, 1000, 5000, 5001])
def test_scaled_sum_with_the_next_norm(width):
    g = torch.Generator().manual_seed(width)
    rnd = lambda *s: torch.randn(*s, generator=g)
    x, a, b, wa, wb, w = 3 * rnd(7, width), rnd(7, width), 2 * rnd(7, width), rnd(width), rnd(width), rnd(width)
    d = lambda t: t.to(DEV)
    y = x.double() + wa.double() * a.double() + wb.double() * b.double()
    xd = d(x)
    out = ops.scaled_sum_norm(xd, d(a), d(wa), d(b), d(wb), d(w), 1e-5, torch.float32)
    assert torch.allclose(xd.double().cpu(), y, rtol=1e-5, atol=1e-5)                     # the sum is kept, in place
    assert torch.allclose(out.double().cpu(), pb.norm(y, w, 1e-5), rtol=1e-5, atol=1e-5)
    half = ops.scaled_sum_norm(d(x), d(a), d(wa), d(b), d(wb), d(w), 1e-5, torch.bfloat16)
    assert torch.equal(half.cpu(), out.cpu().to(torch.bfloat16))
    # picked rows: nothing is stored
    xd = d(x)
    rows = torch.tensor([3, 0, 3], dtype=torch.int32, device=DEV)
    picked = ops.scaled_sum_norm(xd, d(a), d(wa), d(b), d(wb), d(w), 1e-5, torch.float32, rows=rows)
    assert torch.equal(xd.cpu(), x) and torch.equal(picked.cpu(), out.cpu()[[3, 0, 3]])
    # one term, and none
    one = ops.scaled_sum_norm(d(x), d(a), d(wa), None, None, d(w), 1e-5, torch.float32)
    assert torch.allclose(one.double().cpu(), pb.norm(x.double() + wa.double() * a.double(), w, 1e-5), rtol=1e-5, atol=1e-5)
    none = ops.scaled_sum_norm(d(x), None, None, None, None, d(w), 1e-5, torch.float32)
    assert torch.allclose(none.double().cpu(), pb.norm(x.double(), w, 1e-5), rtol=1e-5, atol=1e-5)


# ----------------------------------------------------------------------------------------------- attention

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("sizes,rot", [
    ((6, 2, 64, 48), {"base": 3000.0, "dims": 64, "scaling": {"factor": 3.0}}), ((3, 3, 10, 7), {"base": 50.0, "dims": 10, "scaling": None}),
    ((2, 1, 13, 12), {"base": 10000.0, "dims": 2, "scaling": {"factor": 0.5}}), ((4, 1, 32, 32), {"base": 1000.0, "dims": 8, "scaling": {"factor": 4.0}}),
    ((12, 2, 128, 128), {"base": 1000.0, "dims": 96, "scaling": {"factor": 4.0}}), ((1, 1, 9, 5), None)])
def test_rotated_unit_heads_and_the_cache_write(dtype, sizes, rot):
    H, G, d, dv = sizes
    eps = 1e-3                                                   # (large: it must be inside the root)
    g = torch.Generator().manual_seed(d)
    lens, pos0 = [21, 1, 6], [13, 127, 0]
    step = _Step(lens, pos0, [0, 1, 2])
    T = sum(lens)
    C = (H + G) * d + G * dv
    rows = (torch.randn(T, C + 5, generator=g) * 0.3).to(dtype)
    table = torch.tensor([[3, 7, 1] + [-1] * 6, [5, 0, 2, 9, 10, 11, 12, 13, 8], [4] + [-1] * 8], dtype=torch.int32, device=DEV)
    kc = torch.full((14, G, 16, d), float("nan"), dtype=dtype, device=DEV)
    vc = torch.full((14, G, 16, dv), float("nan"), dtype=dtype, device=DEV)
    cos = sin = None
    n_rot = 0
    if rot is not None:
        ang = torch.arange(200, dtype=F)[:, None] * pb.frequencies(rot["dims"], rot["base"], (rot["scaling"] or {"factor": 1.0})["factor"])[None, :]
        cos, sin, n_rot = torch.cos(ang).float().to(DEV), torch.sin(ang).float().to(DEV), rot["dims"]
    args = (cos, sin, n_rot, 0.0, 0, False, step, table)
    q_out = ops.head_prepare(rows.to(DEV), 3, None, None, eps, *args, kc, vc, H, G, d, dv, True, unit_norm=True, layout="half")
    assert int(step.status.item()) == 0
    pos = step.positions.cpu().long()
    r = rows.double()
    q, k = r[:, 3:3 + H * d].view(T, H, d), r[:, 3 + H * d:3 + (H + G) * d].view(T, G, d)
    v = r[:, 3 + (H + G) * d:3 + C].view(T, G, dv)
    turn = (lambda x: pb.rms(pb.rotate_halves(x, pos, rot), eps)) if rot is not None else (lambda x: pb.rms(x, eps))     # rotation first
    assert torch.allclose(q_out.double().cpu().view(T, H, d), turn(q), **_tol(dtype))
    seg = step.token_seg.cpu().tolist()
    for t in range(T):
        page, place = int(table[seg[t], int(pos[t]) // 16]), int(pos[t]) % 16
        assert torch.allclose(kc[page, :, place].double().cpu(), turn(k)[t], **_tol(dtype))
        assert torch.equal(vc[page, :, place].cpu(), v[t].to(dtype))
    assert int(torch.isnan(kc.float()).sum()) == (14 * 16 - T) * G * d            # nothing else was written
    # a layer that reads another's pages: rows of queries alone, the same bits, no write
    only_q = torch.cat([rows[:, :3 + H * d], rows[:, -1:]], dim=1).contiguous()
    kc2 = torch.full_like(kc, float("nan"))
    q2 = ops.head_prepare(only_q.to(DEV), 3, None, None, eps, *args, kc2, vc, H, G, d, dv, False, unit_norm=True, layout="half", own_kv=False)
    assert torch.equal(q2, q_out) and bool(torch.isnan(kc2.float()).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("H,dv", [(3, 7), (6, 64), (2, 128)])
def test_a_gate_per_head(H, dv, dtype):
    g = torch.Generator().manual_seed(dv)
    ctx, rows = torch.randn(5, H * dv, generator=g).to(dtype), torch.randn(5, H + 4, generator=g).to(dtype)
    got = ops.gate_mul(ctx.to(DEV), rows.to(DEV), 2, dv)
    want = (ctx.double().view(5, H, dv) * torch.sigmoid(rows.double()[:, 2:2 + H])[:, :, None]).view(5, -1)
    assert torch.allclose(got.double().cpu(), want, **_tol(dtype))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("window,keep", [(None, 0), (5, 2), (96, 20), (150, 130), (40, 200)])
def test_single_tokens_with_kept_keys_and_a_gate_per_head(window, keep, dtype):
    """Keys at both edges of the window and of the kept keys stand out; the merge applies the gate, with the bits of the
    gate's own kernel."""
    H, G, d, dv = 6, 2, 24, 40
    n, scale = 420, 0.3
    g = torch.Generator().manual_seed((window or 0) + keep)
    q = pb.rms(torch.randn(n, H, d, generator=g, dtype=F), 1e-6).to(dtype).double()
    k = pb.rms(torch.randn(n, G, d, generator=g, dtype=F), 1e-6)
    v = torch.randn(n, G, dv, generator=g).to(dtype).double()
    probes = [0, 1, 15, 16, 127, 128, 129, 255, 300, 383, 384, 419]
    for i, pr in enumerate(probes):
        for j, h in ((pr - (window or 1) + 1, 0), (pr - (window or 1), 1), (keep - 1, 2), (keep, 4)):
            if 0 <= j <= pr:
                k[j, h // 3] += 2.0 * q[pr, h]
    k = k.to(dtype).double()
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(3, dim=1)) * scale
    w = torch.softmax(s.masked_fill(~pb.visible(n, window, keep)[None], -math.inf), dim=-1)
    want = torch.einsum("hij,jhd->ihd", w, v.repeat_interleave(3, dim=1))[probes]
    table_row = list(np.random.default_rng(1).permutation(30))[:27]
    kc, vc = _paged([k], [v], [table_row], 30, G, d, dv, dtype)
    table = torch.tensor([table_row] * len(probes), dtype=torch.int32, device=DEV)
    step = _Step([1] * len(probes), probes, list(range(len(probes))))
    step.seg_lens, step.max_q_len, step.max_ctx_len = step.lens, 1, n
    rows = q[probes].reshape(-1, H * d).to(dtype).to(DEV).contiguous()
    gate = torch.randn(len(probes), 3 + H, generator=g).to(dtype).to(DEV)
    run = lambda **kw: ops.attention_split(rows, kc.to(DEV), vc.to(DEV), table, step, H, G, d, dv, window, scale, keep_first=keep, **kw)
    plain = run()
    assert torch.allclose(plain.double().cpu().view(-1, H, dv), want, **_tol(dtype))
    assert torch.equal(run(gate=gate, gate_col=3, gate_per_head=True), ops.gate_mul(plain.clone(), gate, 3, dv))


# ----------------------------------------------------------------------------------------------- state space layers

@pytest.mark.parametrize("sizes", [(4, 16, 24, 2, 4), (3, 7, 5, 1, 2), (6, 3, 33, 3, 1), (2, 24, 16, 1, 7)])
def test_filter_steps_and_decays_over_steps(sizes):
    """Filters of one to seven taps over unequal segments, down to single tokens that move their own tails."""
    H, dv, N, G, taps = sizes
    C = H * dv + 2 * G * N
    g = torch.Generator().manual_seed(C)
    seqs = {s: torch.randn(n, 3 + C + H, generator=g) for s, n in ((0, 46), (2, 25))}
    fw, fb, dtb, al = torch.randn(C, taps, generator=g), torch.randn(C, generator=g), torch.randn(H, generator=g), torch.randn(H, generator=g)
    seqs[0][5, 3 + C:] = 50.0                                          # far beyond where softplus is its argument
    seqs[0][6, 3 + C:] = -50.0
    ref = {}
    for s, r in seqs.items():
        dt = pb.softplus(r[:, 3 + C:].double() + dtb.double())
        ref[s] = (pb.silu(pb.causal_filter(r[:, 3:3 + C].double(), fw, fb)), torch.exp(-torch.exp(al.double()) * dt), dt)
    tails = torch.full((3, max(1, taps - 1), C), float("nan"), device=DEV) if taps > 1 else None
    if tails is not None:
        tails[0].zero_(), tails[2].zero_()
    at = {0: 0, 2: 0}
    d = lambda t: t.to(DEV).contiguous()
    for lens in ([1, 2], [2, 1], [17, 9], [1, 1], [1, 1], [24, 11]):
        step = _Step(lens, [at[0], at[2]], [0, 2])
        rows = d(torch.cat([seqs[s][at[s]:at[s] + m] for s, m in zip((0, 2), lens)]))
        single = max(lens) == 1 and taps > 1
        out, g_col = ops.filter_prepare(rows, 3, d(fw.t()), d(fb), tails, 3 + C, d(dtb), d(al), step, single)
        if tails is not None and not single:
            ops.tail_update(rows, 3, tails, step.seg_start, step.seg_slot)
        want = [torch.cat([ref[s][i][at[s]:at[s] + m] for s, m in zip((0, 2), lens)]) for i in range(3)]
        for got, w in zip((out[:, :C], out[:, g_col:g_col + H], out[:, g_col + H:g_col + 2 * H]), want):
            assert torch.allclose(got.double().cpu(), w, rtol=2e-5, atol=2e-5)
        for s, m in zip((0, 2), lens):
            at[s] += m
    if tails is not None:
        assert bool(torch.isnan(tails[1]).all())
        assert torch.equal(tails[0].cpu(), seqs[0][46 - taps + 1:, 3:3 + C])


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5])
def test_filter_over_prompt_portions_and_single_tokens_has_the_same_bits(taps):
    """Long segments (several tokens a thread), a boundary inside a thread's tokens, and the same tokens in short steps."""
    H, dv, N, G = 2, 12, 8, 1
    C = H * dv + 2 * G * N
    g = torch.Generator().manual_seed(taps)
    n = (203, 130)
    seqs = [torch.randn(m, C + H + 2, generator=g) for m in n]
    fw, fb, dtb, al = torch.randn(C, taps, generator=g), torch.randn(C, generator=g), torch.randn(H, generator=g), torch.randn(H, generator=g)
    d = lambda t: t.to(DEV).contiguous()

    def run(cuts):
        tails = torch.zeros(2, max(1, taps - 1), C, device=DEV) if taps > 1 else None
        at, outs = [0, 0], [[], []]
        for lens in cuts:
            step = _Step(lens, list(at), [0, 1])
            rows = d(torch.cat([s[a:a + m] for s, a, m in zip(seqs, at, lens)]))
            out, g_col = ops.filter_prepare(rows, 0, d(fw.t()), d(fb), tails, C, d(dtb), d(al), step)
            if tails is not None:
                ops.tail_update(rows, 0, tails, step.seg_start, step.seg_slot)
            out = out[:, :g_col + 3 * H].cpu()
            outs[0].append(out[:lens[0]]), outs[1].append(out[lens[0]:])
            at = [a + m for a, m in zip(at, lens)]
        return [torch.cat(o) for o in outs]
    whole, cut = run([[203, 130]]), run([[100, 65], [101, 1], [2, 64]])
    for s in range(2):
        assert torch.equal(whole[s], cut[s])
        y = pb.silu(pb.causal_filter(seqs[s][:, :C].double(), fw, fb))
        dt = pb.softplus(seqs[s][:, C:C + H].double() + dtb.double())
        lng = -torch.exp(al.double()) * dt
        want = torch.cat([y, torch.exp(lng), dt, lng], dim=1)
        assert torch.allclose(whole[s].double(), want, rtol=2e-5, atol=2e-5)


SCAN_SIZES = [(2, 2, 16, 32), (4, 2, 40, 20), (3, 1, 5, 9), (2, 1, 128, 64), (4, 4, 8, 4), (2, 2, 160, 128), (1, 1, 33, 3), (6, 3, 64, 24)]


def _step_case(H, G, d, dv, seed, lens):
    g = torch.Generator().manual_seed(seed)
    out = {}
    for s, n in zip((0, 2), lens):
        out[s] = {"q": torch.randn(n, G, d, generator=g), "k": torch.randn(n, G, d, generator=g) * 0.5, "v": torch.randn(n, H, dv, generator=g),
                  "g": torch.rand(n, H, generator=g) ** 0.2, "b": torch.rand(n, H, generator=g)}
        out[s]["g"][n // 2] = 0.0                                          # a token that forgets everything
        out[s]["g"][n // 3] = 1e-30
    return out


def _step_rows(seqs, at, lens):
    parts, aux = [], []
    for s, m in zip((0, 2), lens):
        x = {k: v[at[s]:at[s] + m].reshape(m, -1) for k, v in seqs[s].items()}
        parts.append(torch.cat([x["q"], x["k"], x["v"]], dim=1))
        aux.append(torch.cat([torch.zeros(m, 1), x["g"], x["b"], torch.log(x["g"])], dim=1))
    rows = torch.cat([torch.zeros(sum(lens), 4), torch.cat(parts)], dim=1)
    return rows.to(DEV).contiguous(), torch.cat(aux).to(DEV).contiguous()


def _step_reference(seqs, H, G, skip):
    ref = {}
    for s, x in seqs.items():
        per = H // G
        dd = {k: v.double() for k, v in x.items()}
        o = [pb.fading_scan(dd["q"][:, h // per], dd["k"][:, h // per], dd["v"][:, h], dd["g"][:, h], dd["b"][:, h], float(skip[h]))[0] for h in range(H)]
        n = [pb.fading_scan(dd["q"][:, h // per], dd["k"][:, h // per], torch.ones(len(x["q"]), 1, dtype=F), dd["g"][:, h], dd["b"][:, h], 0.0)[0][:, 0]
             for h in range(H)]
        ref[s] = (torch.stack(o, dim=1), torch.stack(n, dim=1))
    return ref


@pytest.mark.parametrize("sizes", SCAN_SIZES)
@pytest.mark.parametrize("ones", [False, True], ids=["values", "ones"])
def test_scan_with_a_decay_and_a_strength_per_token_over_steps(sizes, ones):
    """With a skip, and with the column of ones that a memory is normalised by; decays of 0 and 1e-30 among them."""
    H, G, d, dv = sizes
    seqs = _step_case(H, G, d, dv, d + dv, (46, 25))
    skip = torch.linspace(-1, 1, H)
    ref = _step_reference(seqs, H, G, skip)
    state = torch.full((3, H, d, dv), float("nan"), device=DEV)
    n_state = torch.full((3, H, d), float("nan"), device=DEV)
    for t in (state, n_state):
        t[0].zero_(), t[2].zero_()
    at = {0: 0, 2: 0}
    for lens in ([1, 2], [2, 1], [17, 9], [1, 1], [25, 12]):
        step = _Step(lens, [at[0], at[2]], [0, 2])
        rows, aux = _step_rows(seqs, at, lens)
        got = ops.state_scan(ops.SCAN_STEP, rows, 4, 4 + G * d, 4 + 2 * G * d, aux, 1, state, step.seg_start, step.seg_slot, H, H // G, d, dv,
                             True, max(lens), bonus=skip.to(DEV), ones_state=n_state if ones else None)
        o, n = got if ones else (got, None)
        want = [torch.cat([ref[s][i][at[s]:at[s] + m] for s, m in zip((0, 2), lens)]) for i in range(2)]
        assert torch.allclose(o.double().cpu().view(-1, H, dv), want[0], rtol=2e-5, atol=5e-5)
        if ones:
            assert torch.allclose(n.double().cpu(), want[1], rtol=2e-5, atol=5e-5)
        for s, m in zip((0, 2), lens):
            at[s] += m
    assert bool(torch.isnan(state[1]).all()) and bool(torch.isnan(n_state).all(dim=-1)[1].all())


@pytest.mark.parametrize("d,dv", [(40, 24), (128, 128), (64, 132), (16, 260), (200, 8), (33, 9)])
def test_step_scan_cuttings_are_bit_equal(d, dv):
    """Whole, in portions, and one token at a time (which has a kernel of its own where a row is whole 16-byte pieces)."""
    H, G, n = 2, 1, 45
    seqs = _step_case(H, G, d, dv, 9, (n, 3))
    outs = []
    for cuts in ([45], [1] * 45, [2] * 22 + [1], [7, 30, 8]):
        state, n_state = torch.zeros((1, H, d, dv), device=DEV), torch.zeros((1, H, d), device=DEV)
        got, at = [], 0
        for m in cuts:
            step = _Step([m], [at], [0])
            rows, aux = _step_rows({0: seqs[0]}, {0: at}, [m])
            o, den = ops.state_scan(ops.SCAN_STEP, rows, 4, 4 + G * d, 4 + 2 * G * d, aux, 1, state, step.seg_start, step.seg_slot, H, H // G, d, dv,
                                    True, m, ones_state=n_state)
            got.append(torch.cat([o, den], dim=1))
            at += m
        outs.append(torch.cat(got).cpu())
    for o in outs[1:]:
        assert torch.equal(o, outs[0])


@pytest.mark.parametrize("sizes", [(2, 2, 16, 32), (4, 2, 40, 20), (3, 1, 5, 9), (2, 1, 128, 64), (24, 2, 128, 128), (5, 1, 33, 3), (6, 3, 64, 24), (12, 12, 64, 128)])
@pytest.mark.parametrize("ones", [False, True], ids=["values", "ones"])
def test_scan_in_chunks_on_the_tensor_cores_over_steps(sizes, ones):
    """Segments around multiples of 64 tokens beside short ones, the state carried from chunked steps to single tokens and
    back; decays of 0 and 1e-30 among them. Inputs are bfloat16 numbers: the chunked form then rounds nothing of them, and
    agrees with the exact recurrence to the sixteen bits that it keeps of states and scores."""
    H, G, d, dv = sizes
    total = (330, 276)
    seqs = _step_case(H, G, d, dv, d + dv, total)
    for x in seqs.values():
        for n in "qkv":
            x[n] = x[n].to(torch.bfloat16).float()
        x["g"][:] = torch.where(x["g"] > 1e-20, x["g"] ** 0.1, x["g"])            # (states that hold many tokens)
    skip = torch.linspace(-1, 1, H)
    ref = _step_reference(seqs, H, G, skip)
    state = torch.full((3, H, d, dv), float("nan"), device=DEV)
    n_state = torch.full((3, H, d), float("nan"), device=DEV)
    for t in (state, n_state):
        t[0].zero_(), t[2].zero_()
    at = {0: 0, 2: 0}
    before = ops.LAUNCH_KINDS["ib_chunk_scan"]
    steps = ([100, 63], [1, 1], [64, 128], [2, 65], [128, 1], [33, 16], [2, 2])
    for lens in steps:
        step = _Step(lens, [at[0], at[2]], [0, 2])
        step.max_q_len = max(lens)
        rows, aux = _step_rows(seqs, at, lens)
        got = ops.step_scan(rows, 4, 4 + G * d, 4 + 2 * G * d, aux, 1, 1 + H, 1 + 2 * H, state, step, H, H // G, d, dv, True,
                            skip=skip.to(DEV), ones_state=n_state if ones else None, chunked=True)
        o, n = got if ones else (got, None)
        want = [torch.cat([ref[s][i][at[s]:at[s] + m] for s, m in zip((0, 2), lens)]) for i in range(2)]
        size = float(want[0].abs().max())
        assert torch.allclose(o.double().cpu().view(-1, H, dv), want[0], rtol=2e-4, atol=4e-5 * size), lens
        if ones:
            assert torch.allclose(n.double().cpu(), want[1], rtol=2e-4, atol=4e-5 * float(want[1].abs().max()))
        for s, m in zip((0, 2), lens):
            at[s] += m
    assert ops.LAUNCH_KINDS["ib_chunk_scan"] - before == sum(max(l) >= ops.CHUNK_SCAN_FROM for l in steps)
    assert (at[0], at[2]) == total and bool(torch.isnan(state[1]).all()) and bool(torch.isnan(n_state[1]).all())


@pytest.mark.parametrize("size,groups", [(7, 3), (24, 1), (64, 2), (768, 2), (2000, 1)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
def test_gate_in_front_of_a_norm_over_groups(size, groups, dtype):
    g = torch.Generator().manual_seed(size)
    o, z, w = torch.randn(6, groups * size, generator=g), torch.randn(6, 5 + groups * size, generator=g), torch.randn(groups * size, generator=g)
    d = lambda t: t.to(DEV)
    got = ops.group_norm_gate(d(o), d(w), 1e-2, d(z), 5, "silu", groups, size, dtype, gate_first=True)
    p = (o.double() * pb.silu(z[:, 5:].double())).view(6, groups, size)
    assert torch.allclose(got.double().cpu(), pb.rms(p, 1e-2).view(6, -1) * w.double(), **_tol(dtype))


# ----------------------------------------------------------------------------------------------- matrix memories

@pytest.mark.parametrize("H,cap", [(3, 2.5), (1, 15.0), (12, 6.0)])
def test_memory_gates_over_steps(H, cap):
    """The running maximum over unequal segments, cuttings bit-equal; the second sequence is longer than a tile."""
    g = torch.Generator().manual_seed(H)
    bi, bf = torch.randn(H, generator=g), 2.0 + torch.randn(H, generator=g)
    seqs = {0: 6 * torch.randn(46, 2 + 2 * H, generator=g), 2: 6 * torch.randn(2225, 2 + 2 * H, generator=g)}
    ref = {}
    for s, r in seqs.items():
        i, f = pb.memory_gates(r[:, 2:2 + H].double() + bi.double(), r[:, 2 + H:].double() + bf.double(), cap)
        m, rows = torch.zeros(H, dtype=F), []
        for t in range(len(r)):
            new = torch.maximum(f[t] + m, i[t])
            rows.append(torch.cat([torch.exp(f[t] + m - new), torch.exp(i[t] - new), torch.exp(-new)]))
            m = new
        ref[s] = torch.stack(rows)
    d = lambda t: t.to(DEV).contiguous()

    def run(all_lens, blocks=False):
        state = torch.full((3, H), float("nan"), device=DEV)
        state[0].zero_(), state[2].zero_()
        at, outs = {0: 0, 2: 0}, {0: [], 2: []}
        for lens in all_lens:
            step = _Step(lens, [at[0], at[2]], [0, 2])
            rows = d(torch.cat([seqs[s][at[s]:at[s] + m] for s, m in zip((0, 2), lens)]))
            step.max_q_len = max(lens)
            got = ops.memory_gates(rows, 2, 2 + H, d(bi), d(bf), cap, state, step, blocks=blocks).cpu()
            assert torch.allclose(got[:, 3 * H:].exp(), got[:, :H], rtol=1e-6)
            got = got[:, :3 * H]
            outs[0].append(got[:lens[0]]), outs[2].append(got[lens[0]:])
            for s, m in zip((0, 2), lens):
                at[s] += m
        assert bool(torch.isnan(state[1]).all())
        return {s: torch.cat(o) for s, o in outs.items()}
    a = run([[1, 2], [2, 1], [17, 9], [1, 1], [25, 2212]])
    b = run([[45, 2224], [1, 1]])
    c, e = run([[45, 2224], [1, 1]], True), run([[1, 3], [33, 65], [12, 2157]], True)
    for s in (0, 2):
        assert torch.allclose(a[s].double(), ref[s], rtol=3e-5, atol=1e-6)
        assert torch.equal(a[s], b[s])
        for x in (c, e):                                     # a block of tokens at a time: up to rounding
            assert torch.allclose(x[s].double(), ref[s], rtol=3e-5, atol=1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("H,dv", [(3, 9), (2, 128), (1, 600)])
def test_normalised_read_out_with_head_norm_and_gate(H, dv, dtype):
    g = torch.Generator().manual_seed(dv)
    T, eps, mult, floor = 6, 1e-3, 0.25, 1e-6
    o, den = torch.randn(T, H * dv, generator=g), torch.randn(T, H, generator=g)
    low = torch.rand(T, 2 + H, generator=g) * 0.3
    den[0], den[1] = 0.0, -5.0
    low[0] = 0.0                                                     # nothing but the constant divides
    z, w = torch.randn(T, 4 + H * dv, generator=g), torch.randn(H * dv, generator=g)
    d = lambda t: t.to(DEV)
    got = ops.group_norm_gate(d(o), d(w), eps, d(z), 4, "sigmoid", H, dv, dtype, den=d(den), den_floor=d(low), floor_col=2, den_mult=mult,
                              den_eps=floor)
    x = mult * o.double().view(T, H, dv) / (torch.maximum((mult * den.double()).abs(), low[:, 2:].double()) + floor)[:, :, None]
    want = pb.rms(x, eps).view(T, -1) * w.double() * torch.sigmoid(z[:, 4:].double())
    assert torch.allclose(got.double().cpu(), want, **_tol(dtype))


# ----------------------------------------------------------------------------------------------- the router

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("E,top,width", [(8, 2, 1536), (4, 4, 8), (9, 1, 264), (16, 4, 40), (33, 3, 512), (64, 6, 1000), (3, 2, 72)])
def test_router_with_its_product(E, top, width, dtype):
    g = torch.Generator().manual_seed(E)
    x, w = torch.randn(37, width, generator=g).to(dtype), (torch.randn(E, width, generator=g) * width ** -0.5 * 2).to(dtype)
    weights, chosen = ops.route_rows(x.to(DEV), w.to(DEV), top, want_chosen=True)
    z = x.double() @ w.double().T
    want, ww, gap = pb.route_top(z, top)
    clear = gap > 1e-4
    assert int(clear.sum()) >= 30
    assert torch.equal(chosen.cpu().long()[clear], want[clear])
    full = torch.zeros(37, E, dtype=F).scatter_(1, want, ww)
    assert torch.allclose(weights.double().cpu()[clear], full[clear], rtol=1e-4, atol=1e-6)
    assert torch.equal(ops.route_rows(x[5:6].to(DEV).contiguous(), w.to(DEV), top)[0][0], weights[5])      # whatever else is in the step
    assert ops.route_rows(torch.zeros(2, 12, device=DEV), torch.zeros(4, 12, device=DEV), 1) is None       # no whole pieces: another path


@pytest.mark.parametrize("T,E,top,width,ff", [(300, 8, 2, 128, 72), (256, 16, 4, 64, 16), (513, 8, 1, 136, 200), (700, 5, 2, 1536, 1120), (2048, 8, 2, 256, 264)])
@pytest.mark.parametrize("with_residual", [False, True])
def test_products_over_rows_grouped_by_expert(T, E, top, width, ff, with_residual):
    """Every pair of a token and a chosen expert has one row; experts without a row, with a few, and with several tiles of rows;
    both grouped products, the gated activation with the token's weight, and the sum over a token's rows."""
    from infer_b200 import fast_ops
    g = torch.Generator().manual_seed(T)
    x = torch.randn(T, width, generator=g).to(torch.bfloat16)
    z = torch.randn(T, E, generator=g) + torch.linspace(4, -4, E)            # (unequal groups)
    z[:, E // 2] = -1e9                                                      # one expert that nobody chose
    chosen, ww, _ = pb.route_top(z.double(), top)
    weights = torch.zeros(T, E, dtype=F).scatter_(1, chosen, ww)
    gu = (torch.randn(2 * E * ff, width, generator=g) * width ** -0.5).to(torch.bfloat16)
    down = (torch.randn(width, E * ff, generator=g) * ff ** -0.5).to(torch.bfloat16)
    groups = fast_ops.RowGroups(weights.float().to(DEV), chosen.int().to(DEV).contiguous())
    n_tiles = int(groups.tiles[0])
    assert n_tiles == sum(-(-int((chosen == e).sum()) // 128) for e in range(E)) <= groups.max_tiles
    place = groups.place.cpu().view(T, top).long()
    assert len(set(place.flatten().tolist())) == T * top
    expert_of = groups.tiles[1:1 + n_tiles].cpu().long()
    assert torch.equal(expert_of[place // 128], chosen) and torch.equal(groups.row_of.cpu()[place].long(), torch.arange(T)[:, None].expand(T, top))
    assert torch.allclose(groups.scale.cpu()[place, 0].double(), ww, rtol=1e-6)
    rows, up = groups.product(groups.gather(x.to(DEV)), gu.to(DEV), ff, 2, 0, torch.bfloat16)
    act = ops.glu_act(rows, 0, up, ff, "swish", 0.0, 0.0, 1.0, groups.scale, ff, 1)
    y, _ = groups.product(act, down.to(DEV), width, 1, 1, torch.float32)
    res = torch.randn(T, width, generator=g) if with_residual else None
    out = groups.combine(y, res.clone().to(DEV) if res is not None else None).double().cpu()
    want = res.double() if res is not None else torch.zeros(T, width, dtype=F)
    for e in range(E):
        at = (chosen == e).nonzero()
        t, w = at[:, 0], ww[at[:, 0], at[:, 1]]
        r = lambda v: v.to(torch.bfloat16).double()
        gate, upv = (r(x[t].double() @ gu[o + e * ff:o + (e + 1) * ff].double().T) for o in (0, E * ff))
        want[t] += r(pb.silu(gate) * upv * w[:, None]) @ down[:, e * ff:(e + 1) * ff].double().T
    assert torch.allclose(out, want, rtol=2e-2, atol=2e-2) and float((out - want).pow(2).mean().sqrt()) < 4e-3
