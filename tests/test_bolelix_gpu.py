"""Bolelix in the engine against the plain implementation: every way of cutting requests into steps, in float32 and
bfloat16, on configurations that differ in every size and option; generation through the Python entry point and
the scheduler; the trace and generation programs."""
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import bolelix_cases as BC
import helpers as H
import plain_bolelix as pb

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16]
SEED = 11


def _engine(case, dtype, max_tokens=1024, **kw):
    """case: a configuration's name, or a configuration."""
    from infer_b200.engine import Engine
    cfg = BC.CASES[case] if isinstance(case, str) else case
    return Engine(BC.spec_of(cfg), BC.make_weights(cfg, SEED, decisive=dtype == torch.bfloat16), dtype=dtype, max_tokens=max_tokens,
                  max_requests=4, **kw)


def _requests(name, lengths, seed0=0):
    return {f"r{i}": BC.random_ids(BC.CASES[name], n, seed0 + i) for i, n in enumerate(lengths)}


@pytest.mark.parametrize("dtype", DTYPES, ids=["f32", "bf16"])
@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_whole(name, dtype):
    reqs = _requests(name, [5, 17, 33, 90, 1, 2])
    eng = _engine(name, dtype)
    got = H.run_trace(eng, H.trace_whole(reqs))
    BC.check(BC.CASES[name], SEED, dtype, got, reqs, what=name)
    assert eng.cache.pages_in_use() == [0] * len(eng.cache.groups)


@pytest.mark.parametrize("dtype", DTYPES, ids=["f32", "bf16"])
@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_tail_one_by_one(name, dtype):
    """The last 40 tokens decoded one by one: windows of 3, 5, 9, 24, 33 and 40 pass over decoded tokens, pages go back."""
    reqs = _requests(name, [110, 47], seed0=10)
    got = H.run_trace(_engine(name, dtype), H.trace_tail(reqs, 40))
    BC.check(BC.CASES[name], SEED, dtype, got, reqs, what=name)


@pytest.mark.parametrize("dtype", DTYPES, ids=["f32", "bf16"])
@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_portions_of_changing_size(name, dtype):
    reqs = _requests(name, [150, 61], seed0=20)
    got = H.run_trace(_engine(name, dtype), H.trace_portions(reqs))
    BC.check(BC.CASES[name], SEED, dtype, got, reqs, what=name)


@pytest.mark.parametrize("dtype", DTYPES, ids=["f32", "bf16"])
@pytest.mark.parametrize("name", ["a", "b"])
def test_mixed_with_pages_and_slots_used_again(name, dtype):
    lengths = [60, 45, 100, 33, 64, 90, 20, 77]
    ids = _requests(name, lengths, seed0=30)
    reqs = {rid: (t, max(2, len(t) - 16 - 3 * i)) for i, (rid, t) in enumerate(ids.items())}
    max_tokens = 320                                        # 20 pages, 4 slots: fewer than the requests need in total
    steps = H.trace_mixed(reqs, max_tokens, seed=7)
    assert max(len(s["entries"]) for s in steps) >= 3
    eng = _engine(name, dtype, max_tokens=max_tokens)
    got = H.run_trace(eng, steps)
    BC.check(BC.CASES[name], SEED, dtype, got, ids, what=name)
    assert sum(-(-n // 16) for n in lengths) > eng.cache.pages_total()[0] and len(lengths) > eng.cache.n_slots
    assert eng.cache.pages_in_use() == [0] * len(eng.cache.groups)


@pytest.mark.parametrize("name", ["a", "b"])
def test_cuttings_are_bit_equal_in_float32(name):
    """Prefill against token-by-token decoding and against portions down to two tokens: the state that a cut carries
    (pages, the row of the token before, state matrices) is exactly what the uncut run had in its registers."""
    reqs = _requests(name, [97], seed0=40)
    dtype = torch.float32
    a = H.run_trace(_engine(name, dtype), H.trace_whole(reqs))["r0"]
    b = H.run_trace(_engine(name, dtype), H.trace_tail(reqs, 96))["r0"]          # one token, then 96 one by one
    c = H.run_trace(_engine(name, dtype), H.trace_portions(reqs))["r0"]
    ids = reqs["r0"]
    bounds = list(range(0, 96, 2)) + [97]                        # portions of two tokens; the last one has three
    twos = [{"entries": [("r0", ids[a:b], list(range(b - a)))], "end": []} for a, b in zip(bounds[:-1], bounds[1:])]
    d = H.run_trace(_engine(name, dtype), twos)["r0"]
    for p in a:
        for other in (b, c, d):
            assert np.array_equal(a[p], other[p]), f"position {p} differs between cuttings in float32"


def test_bfloat16_cuttings_differ_by_rounding_only():
    name = "c"
    reqs = _requests(name, [200], seed0=41)
    a = H.run_trace(_engine(name, torch.bfloat16), H.trace_whole(reqs))["r0"]
    b = H.run_trace(_engine(name, torch.bfloat16), H.trace_portions(reqs))["r0"]
    ref = BC.oracle(BC.CASES[name], SEED, torch.bfloat16, reqs["r0"])
    noise = float(np.sqrt(np.mean((BC.oracle(BC.CASES[name], SEED, torch.bfloat16, reqs["r0"], torch.bfloat16) - ref) ** 2)))
    for p in a:
        assert float(np.sqrt(np.mean((a[p] - b[p]) ** 2))) <= 4 * noise


@pytest.mark.parametrize("dtype", DTYPES, ids=["f32", "bf16"])
@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_sharp_attention_at_window_edges_and_page_borders(name, dtype):
    """Peaked attention weights: a position's result hangs on single keys: the farthest in its window, a kept first one, a
    key hundreds of positions back (the layers without a mask). Prompts end and decoding starts around page borders
    (multiples of 16), key chunks (multiples of 128) and where the windows of 150 and 100 begin to pass the kept keys."""
    cfg, sharp = BC.CASES[name], BC.sharpened(BC.CASES[name], 2.5)
    ids = BC.random_ids(cfg, 64, 50)
    flat, peaked = (BC.oracle(c, SEED, torch.float32, ids) for c in (cfg, sharp))
    assert np.abs(flat - peaked).max() > 3e-2 * np.abs(flat).max()                        # the sharpening changes the function
    for n, head in ((337, 303), (320, 289), (321, 288), (200, 155)):
        ids = BC.random_ids(cfg, n, 51 + n)
        steps = [{"entries": [("x", ids[:head], list(range(0, head, 7)) + [head - 1])], "end": []}]
        steps += [{"entries": [("x", [ids[i]], [0])], "end": []} for i in range(head, n)]
        got = H.run_trace(_engine(sharp, dtype), steps)
        BC.check(sharp, SEED, dtype, got, {"x": ids}, what=f"{name}/{n}")


@pytest.mark.parametrize("change", ["window", "keep", "last_kept"])
def test_the_checks_would_notice_a_window_or_a_kept_key_one_off(change):
    """The plain implementation with a window, or a number of kept keys, that is off by one differs from the engine by far
    more than the comparisons allow."""
    sharp = BC.sharpened(BC.CASES["a"], 2.5)
    wrong = BC.sharpened(sharp, 1.0)
    mask = wrong["layers"][1]["mixer"]["mask"]
    if change == "window":
        mask["size"] += 1
    else:
        mask["keep_first"] += 1 if change == "keep" else -1
    ids = BC.random_ids(sharp, 90, 5)
    got = np.stack([v for _, v in sorted(H.run_trace(_engine(sharp, torch.float32), H.trace_whole({"x": ids}))["x"].items())])
    right, off = (BC.oracle(c, SEED, torch.float32, ids) for c in (sharp, wrong))
    assert np.abs(got - off).max() > 50 * np.abs(got - right).max()


def test_tokens_far_back_reach_the_logits():
    """Changing the first token changes logits 300 positions later (through kept keys and the
    recurrences), by the same amount in the engine as in the plain implementation."""
    name = "a"
    cfg = BC.CASES[name]
    ids = BC.random_ids(cfg, 300, 77)
    other = [(ids[0] + 1) % cfg["vocab"]] + ids[1:]
    want = BC.oracle(cfg, SEED, torch.float32, other)[-1] - BC.oracle(cfg, SEED, torch.float32, ids)[-1]
    assert np.abs(want).max() > 1e-4
    eng = _engine(name, torch.float32)
    got = H.run_trace(eng, H.trace_portions({"p": ids, "q": other}))
    assert np.allclose(got["q"][299] - got["p"][299], want, atol=2e-5)


@pytest.mark.parametrize("dtype", DTYPES, ids=["f32", "bf16"])
def test_long_decode(dtype):
    name = "b"
    ids = BC.random_ids(BC.CASES[name], 300, 60)
    steps = [{"entries": [("x", ids[:7], [6])], "end": []}]
    steps += [{"entries": [("x", [ids[i]], [0])], "end": []} for i in range(7, 300)]
    got = H.run_trace(_engine(name, dtype), steps)
    BC.check(BC.CASES[name], SEED, dtype, got, {"x": ids}, what=name)


@pytest.mark.parametrize("dtype", DTYPES, ids=["f32", "bf16"])
@pytest.mark.parametrize("name", ["a", "b"])
def test_first_tokens_one_by_one(name, dtype):
    """From position 0: filters see zeros, states start from zero and the running maximum at zero, the first query's softmax
    holds itself alone."""
    ids = BC.random_ids(BC.CASES[name], 7, 70)
    steps = [{"entries": [("x", [t], [0])], "end": []} for t in ids]
    got = H.run_trace(_engine(name, dtype), steps)
    BC.check(BC.CASES[name], SEED, dtype, got, {"x": ids}, what=name)


def test_a_batch_of_unequal_requests_equals_each_alone():
    name = "b"
    reqs = _requests(name, [3, 90, 41, 2], seed0=80)
    eng = _engine(name, torch.float32)
    alone = H.run_trace(eng, H.trace_whole(reqs))
    together = H.run_trace(eng, [{"entries": [(r, t, list(range(len(t)))) for r, t in reqs.items()], "end": list(reqs)}])
    for r in reqs:
        for p in alone[r]:
            assert np.array_equal(alone[r][p], together[r][p])


def test_long_prompts_run_chunked_scans_and_grouped_experts():
    """A prompt of 300 tokens, and the same tokens in portions: the scans take 64 tokens at a time, routed layers with few chosen
    experts gather their rows; results as for every other way of running them."""
    from infer_b200 import ops
    cfg = BC.CASES["c"]
    ids = BC.random_ids(cfg, 420, 91)
    before = dict(ops.LAUNCH_KINDS)
    got = H.run_trace(_engine("c", torch.bfloat16), [{"entries": [("x", ids[:300], list(range(300)))], "end": []},
                                                     {"entries": [("x", ids[300:], list(range(120)))], "end": ["x"]}])
    ran = {k: v - before.get(k, 0) for k, v in ops.LAUNCH_KINDS.items() if v != before.get(k, 0)}
    assert ran.get("ib_chunk_scan", 0) == 8 and ran.get("ib_group_rows", 0) >= 2 and ran["ib_gemm_tc_grouped"] == 2 * ran["ib_group_rows"], ran
    BC.check(cfg, SEED, torch.bfloat16, got, {"x": ids}, what="long")


def test_the_design_runs_on_its_own_kernels():
    from infer_b200 import ops
    eng = _engine("c", torch.bfloat16)
    ids = BC.random_ids(BC.CASES["c"], 140, 90)
    before = dict(ops.LAUNCH_KINDS)
    H.run_trace(eng, [{"entries": [("x", ids[:139], [138])], "end": []}, {"entries": [("x", ids[139:], [0])], "end": ["x"]}])
    ran = {k: v - before.get(k, 0) for k, v in ops.LAUNCH_KINDS.items() if v != before.get(k, 0)}
    for kind in ("ib_scaled_sum_norm", "ib_filter_prepare", "ib_memory_gates", "ib_group_norm_gate", "ib_head_prepare", "ib_route_rows", "ib_glu_act"):
        assert ran.get(kind, 0) >= 2, (kind, ran)
    assert ran.get("ib_gemm_tc", 0) >= 1                     # the tensor-core product serves the prompt's matrices
    # keys and values of 64 and 128: the prompt's attention runs on the tensor-core kernel, every decoded token's on the
    # kernel that splits its keys over CTAs, none on the plain one
    assert ran.get("ib_attention_prefill_tc_kept", 0) + ran.get("ib_attention_prefill_tc_biased", 0) == 3, ran
    assert ran.get("ib_attention_split", 0) == 3 and "ib_attention_plain" not in ran, ran


# ----------------------------------------------------------------------------------------------- generation, programs

@pytest.mark.parametrize("name", ["a", "b"])
def test_greedy_generation_through_the_scheduler(name):
    from infer_b200.engine.generation import LLM
    cfg = BC.CASES[name]
    prompts = [BC.random_ids(cfg, n, 100 + n) for n in (5, 17, 33, 1)]
    llm = LLM(None, dtype=torch.float32, spec=BC.spec_of(cfg), weights=BC.make_weights(cfg, SEED), slots=3, max_seq=128,
              max_batch_tokens=24)
    outs = llm.generate(prompts, max_new=12)
    W = H.as_compute(BC.make_weights(cfg, SEED), torch.float32)
    for p, o in zip(prompts, outs):
        assert o == pb.greedy(cfg, W, p, 12)
    assert llm.engine.cache.pages_in_use() == [0] * len(llm.engine.cache.groups)


def test_bfloat16_generation_with_graphs_picks_the_maximum_up_to_rounding():
    from infer_b200.engine.generation import LLM
    name = "a"
    cfg = BC.CASES[name]
    prompts = [BC.random_ids(cfg, n, 200 + n) for n in (9, 40, 70)]
    llm = LLM(None, dtype=torch.bfloat16, spec=BC.spec_of(cfg), weights=BC.make_weights(cfg, SEED, decisive=True), slots=4, max_seq=128)
    outs = llm.generate(prompts, max_new=24)
    for p, o in zip(prompts, outs):
        assert len(o) == 24
        ids = p + o
        ref = BC.oracle(cfg, SEED, torch.bfloat16, ids)
        refr = BC.oracle(cfg, SEED, torch.bfloat16, ids, torch.bfloat16)
        noise = max(float(np.sqrt(np.mean((refr - ref) ** 2))), 1e-3 * float(np.sqrt(np.mean(ref ** 2))))
        for i, tok in enumerate(o):
            row = ref[len(p) + i - 1]
            assert row[tok] >= row.max() - 12 * noise, f"token {i}: chose a logit {row.max() - row[tok]:.4f} below the maximum"


def _write_model(folder, cfg, W):
    import json
    from infer_b200.weights import write_safetensors
    os.makedirs(folder)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), W)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program_on_a_model_folder(tmp_path, dtype):
    """bin/trace_run on a written folder."""
    cfg = BC.CASES["a"]
    model = tmp_path / "model"
    _write_model(str(model), cfg, BC.make_weights(cfg, SEED, decisive=dtype == "bfloat16"))
    lengths = [70, 40, 100, 33, 64]
    ids = {f"r{i}": BC.random_ids(cfg, n, 600 + i) for i, n in enumerate(lengths)}
    steps = H.trace_mixed({rid: (t, max(2, len(t) - 20)) for rid, t in ids.items()}, 256, seed=3)
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype", dtype,
                           "--out", str(out), "--max-tokens", "256"], input=H.trace_to_jsonl(steps), capture_output=True,
                          text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    got, pos = {}, {}
    for i, st in enumerate(steps):
        arr = np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
        r = 0
        for rid, toks, want in st["entries"]:
            for w in want:
                got.setdefault(rid, {})[pos.get(rid, 0) + w] = arr[r]
                r += 1
            pos[rid] = pos.get(rid, 0) + len(toks)
    BC.check(cfg, SEED, torch.float32 if dtype == "float32" else torch.bfloat16, got, ids, what="program")


def test_generate_program_on_a_model_folder_and_on_a_preset(tmp_path):
    cfg = BC.CASES["a"]
    model = tmp_path / "model"
    _write_model(str(model), cfg, BC.make_weights(cfg, SEED))
    prompt = BC.random_ids(cfg, 21, 1)
    want = pb.greedy(cfg, H.as_compute(BC.make_weights(cfg, SEED), torch.float32), prompt, 10)
    gen = os.path.join(ROOT, "bin", "generate")

    def run(args):
        proc = subprocess.run([sys.executable, gen] + args, capture_output=True, text=True, timeout=900, cwd=ROOT)
        assert proc.returncode == 0, (proc.stdout[-1500:], proc.stderr[-1500:])
        line = next(l for l in proc.stdout.splitlines() if l.startswith("ids:"))
        return [int(t) for t in line.split()[1:]]
    ids = ",".join(map(str, prompt))
    assert run(["0", "10", "--model", str(model), "--dtype", "float32", "--prompt-ids", ids, "--max-seq", "64"]) == want
    assert run(["0", "10", "--model", str(model), "--dtype", "float32", "--prompt-ids", ids, "--max-seq", "64", "--chunk", "5",
                "--kv-blocks", "3"]) == want
    assert len(run(["0", "12", "--random", "tiny-bolelix", "--max-seq", "64"])) == 12
