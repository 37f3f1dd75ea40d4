"""Lasizen on the device against the plain implementation (``plain_lasizen``): every mechanism
alone, whole prompts against token-by-token decoding, portions down to two tokens, batches of
unequal requests, pages and slots used again, keys just inside and just outside a window in prompts
and decoded, far tokens of the recurrent layers, the first tokens of a sequence, long decoding
through CUDA graphs, other sizes, greedy generation through the entry point, and the kernels alone."""
import json
import os
import random

import numpy as np
import pytest
import torch

import plain_lasizen as plain
import replay
import tiny_lasizen as tl

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64
_folders: dict = {}
_expected: dict = {}


def folder(tmp_path_factory, name, cfg, dtype, tensors=None):
    key = (name, dtype)
    if key not in _folders:
        path = str(tmp_path_factory.mktemp(f"lasizen_{name}_{dtype}"))
        _folders[key] = tl.write_folder(path, cfg, seed=len(name), storage=DTYPES[dtype],
                                        tensors=tensors)
    return _folders[key]


def stored(model_dir):
    """The folder's tensors as float64 (what the file holds, not what was drawn)."""
    from ginfer_b200.weights.safetensors_io import open_model_tensors
    out = {}
    for n, (f, k) in open_model_tensors(model_dir).items():
        t = f.get(k)
        out[n] = t.double() if t.is_floating_point() else t
    return out


def prompts(vocab, lengths, seed=0):
    rng = random.Random(seed)
    return {f"r{i}": [rng.randrange(vocab) for _ in range(n)] for i, n in enumerate(lengths)}


def expected(model_dir, cfg, requests, **kw):
    out = {}
    W = None
    for rid, toks in requests.items():
        key = (model_dir, tuple(toks), tuple(sorted(kw.items())))
        if key not in _expected:
            W = W or stored(model_dir)
            _expected[key] = plain.forward(cfg, W, toks, **kw).numpy()
        out[rid] = _expected[key]
    return out


def make_runner(model_dir, dtype, max_tokens, page_size=16, eager=True, max_live=4):
    from ginfer_b200.engine.loading import load_model
    from ginfer_b200.engine.runner import ModelRunner
    model, _ = load_model(model_dir, dtype, "cuda:0")
    budget = -(-max_tokens // 64) * 64
    return ModelRunner(model, page_size=page_size, max_num_seqs=max_live, max_seq_len=budget,
                       num_pages=budget // page_size, max_num_batched_tokens=budget,
                       enforce_eager=eager)


def rel(row, ref):
    d = row.astype(np.float64) - ref
    d = d - d.mean()
    return float(np.sqrt((d * d).mean()) / np.sqrt(((ref - ref.mean()) ** 2).mean()))


def row_errors(rows, want):
    """Per row: rms of the difference (mean taken off) over the rms of the expected logits."""
    worst, where, errs = 0.0, None, []
    for (rid, pos), row in sorted(rows.items()):
        e = rel(row, want[rid][pos])
        errs.append(e)
        if not e <= worst:
            worst, where = e, (rid, pos)
    return worst, where, float(np.mean(errs)), errs


# float32: differences of summation order.  bfloat16: the folders' peaked attention amplifies the
# format's rounding, so single rows may be off (at most one in thirty) while the mean stays small;
# a misplaced page, a lost state or a window off by one puts most rows near one.
LIMIT = {"float32": (5e-5, 1e-5), "bfloat16": (0.1, 0.02)}


def check(rows, want, dtype, requests):
    assert len(rows) == sum(len(t) for t in requests.values()), "a logits row is missing"
    worst, where, mean, errs = row_errors(rows, want)
    if dtype == "bfloat16":
        over = sum(e > LIMIT[dtype][0] for e in errs)
        assert over <= len(errs) // 30, f"{over} of {len(errs)} rows are off; worst {where}: {worst:.3e}"
    else:
        assert worst <= LIMIT[dtype][0], f"worst row {where}: relative error {worst:.3e}"
    assert mean <= LIMIT[dtype][1], f"mean relative error {mean:.3e}"


# ----------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("name", ["DELTA_ONLY", "ATTENTION_ONLY", "DENSE_FF", "LOOPED"])
def test_each_mechanism_alone(tmp_path_factory, name):
    cfg = getattr(tl, name)
    d = folder(tmp_path_factory, name, cfg, "float32")
    reqs = prompts(cfg["vocab"], [70, 3, 1])
    for steps in (replay.cut_whole(reqs), replay.cut_portions(reqs)):
        rows = replay.run_in_process(make_runner(d, "float32", replay.peak_tokens(steps)), steps)
        check(rows, expected(d, cfg, reqs), "float32", reqs)


@pytest.mark.parametrize("without", ["shift", "norm_b", "loop", "conv", "beta", "decay", "gate", "rot",
                                     "yarn", "qk_norm", "sink", "window"])
def test_the_oracle_without_a_mechanism_is_far_from_the_oracle(tmp_path_factory, without):
    """Passing the comparisons means the mechanism was computed: leaving it out moves the logits by
    much more than any limit."""
    cfg = tl.MIXED
    d = folder(tmp_path_factory, "MIXED", cfg, "float32")
    reqs = prompts(cfg["vocab"], [90], seed=11)
    full = expected(d, cfg, reqs)["r0"]
    less = expected(d, cfg, reqs, without=(without,))["r0"]
    rows = {("r0", p): less[p].astype(np.float32) for p in range(40, 90)}
    assert row_errors(rows, {"r0": full})[2] > 0.01        # the float32 limit is 1e-4


# ----------------------------------------------------------------------------- cuts of the same work
LENGTHS = [150, 97, 41, 5, 1, 66]


def cuts(reqs):
    mixed, _ = replay.cut_mixed(reqs, seed=3, decode_tail=20)
    singles, _ = replay.cut_mixed(reqs, seed=5, decode_tail=9, singles_first=True,
                                  sizes=(2, 2, 3, 17, 40))
    # portions long enough for the tensor-core prompt kernels beside single tokens, in both orders
    long_a, _ = replay.cut_mixed(reqs, seed=9, decode_tail=10, singles_first=True,
                                 sizes=replay.LONG_SIZES)
    long_b, _ = replay.cut_mixed(reqs, seed=10, decode_tail=6, sizes=(64, 80, 65))
    return {"whole": replay.cut_whole(reqs), "decode": replay.cut_tail_decode(reqs, tail=40),
            "portions": replay.cut_portions(reqs), "mixed": mixed, "mixed_singles_first": singles,
            "mixed_long_singles_first": long_a, "mixed_long": long_b}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["MIXED", "OTHER", "WIDE", "ODD"])
def test_cuts_agree_with_plain(tmp_path_factory, name, dtype):
    cfg = getattr(tl, name)
    d = folder(tmp_path_factory, name, cfg, dtype)
    reqs = prompts(cfg["vocab"], LENGTHS, seed=1)
    want = expected(d, cfg, reqs)
    got = {}
    for cut, steps in cuts(reqs).items():
        # the pool holds what the live requests hold and no more: pages and slots are used again
        runner = make_runner(d, dtype, replay.peak_tokens(steps), page_size=8 if name == "OTHER" else 16)
        got[cut] = replay.run_in_process(runner, steps)
        check(got[cut], want, dtype, reqs)
    # how the work was cut changes the logits by rounding only
    for cut in got:
        for key, row in got[cut].items():
            ref = got["whole"][key]
            scale = float(np.abs(ref - ref.mean()).max())
            if dtype == "float32":
                assert float(np.abs(row - ref).max()) <= 1e-3 * scale, (cut, key)


@pytest.mark.parametrize("name", ["MIXED", "OTHER"])
def test_the_first_tokens_of_a_sequence(tmp_path_factory, name):
    """Positions 0, 1, 2: nothing before the first token for shift and convolution, an empty state,
    one key beside the sink; as a prompt of their own, as the start of a longer one, one by one, and
    behind another request that left its slot and pages."""
    cfg = getattr(tl, name)
    d = folder(tmp_path_factory, name, cfg, "float32")
    reqs = prompts(cfg["vocab"], [50, 3, 2, 1], seed=21)
    want = expected(d, cfg, reqs)
    for steps in (replay.cut_whole(reqs), replay.cut_tail_decode(reqs, tail=60),
                  replay.cut_portions(reqs, sizes=(1, 2, 1, 1, 40))):
        runner = make_runner(d, "float32", 64, max_live=1)
        rows = replay.run_in_process(runner, steps)
        check(rows, want, "float32", reqs)
        for rid in reqs:
            for p in range(min(3, len(reqs[rid]))):
                assert rel(rows[(rid, p)], want[rid][p]) <= 1e-4, (rid, p)


@pytest.mark.parametrize("name, dtype", [("MIXED", "float32"), ("WIDE", "bfloat16")])
def test_long_decoding_past_windows_and_pages_through_graphs(tmp_path_factory, name, dtype):
    cfg = getattr(tl, name)
    d = folder(tmp_path_factory, name, cfg, dtype)
    reqs = prompts(cfg["vocab"], [230], seed=2)
    steps = replay.cut_tail_decode(reqs, tail=200)       # 30 in one step, then 200 single tokens
    runner = make_runner(d, dtype, replay.peak_tokens(steps), eager=False)
    check(replay.run_in_process(runner, steps), expected(d, cfg, reqs), dtype, reqs)
    assert runner.graph_launches > 0


def test_decoded_batches_of_many_sizes_through_graphs(tmp_path_factory):
    """Five requests decode together, fewer and fewer as they end, in batches whose graphs are
    padded with rows that belong to no request; slots and pages go to later requests."""
    cfg = tl.MIXED
    d = folder(tmp_path_factory, "MIXED", cfg, "float32")
    reqs = prompts(cfg["vocab"], [60, 45, 70, 52, 66, 49, 58, 40, 63, 71, 44, 56], seed=41)
    steps, at, waiting, live = [], {}, list(reqs), []
    while waiting or live:
        while waiting and len(live) < 10:
            live.append(waiting.pop(0))
        entries = []
        for rid in live:
            n = 30 if at.get(rid, 0) == 0 else 1
            p = at.get(rid, 0)
            entries.append({"id": rid, "tokens": reqs[rid][p:p + n], "want": list(range(n))})
            at[rid] = p + n
        end = [rid for rid in live if at[rid] == len(reqs[rid])]
        live = [rid for rid in live if rid not in end]
        steps.append({"step": len(steps), "entries": entries, "end": end})
    runner = make_runner(d, "float32", replay.peak_tokens(steps), eager=False, max_live=10)
    rows = replay.run_in_process(runner, steps)
    check(rows, expected(d, cfg, reqs), "float32", reqs)
    assert len([k for k in runner._graphs if not isinstance(k[0], str)]) >= 3


@pytest.mark.parametrize("name", ["WIDE", "MIXED"])
def test_equal_prompts_replay_a_graph_of_the_whole_step(tmp_path_factory, name):
    """Prompts of one length, one a step: from the second on the step is captured and replayed, then
    decoded tokens follow; pages and slots are used again."""
    cfg = getattr(tl, name)
    d = folder(tmp_path_factory, name, cfg, "bfloat16")
    reqs = prompts(cfg["vocab"], [300, 300, 300, 300], seed=31)
    steps = []
    for rid, toks in reqs.items():
        steps.append({"step": len(steps), "end": [], "entries": [
            {"id": rid, "tokens": toks[:288], "want": list(range(288))}]})
        for i in range(288, 300):
            steps.append({"step": len(steps), "end": [rid] if i == 299 else [], "entries": [
                {"id": rid, "tokens": [toks[i]], "want": [0]}]})
    runner = make_runner(d, "bfloat16", replay.peak_tokens(steps), eager=False)
    rows = replay.run_in_process(runner, steps)
    check(rows, expected(d, cfg, reqs), "bfloat16", reqs)
    assert any(isinstance(k[0], str) for k in runner._graphs), "no portion step was captured"


def test_trace_program(tmp_path_factory, tmp_path):
    cfg = tl.OTHER
    d = folder(tmp_path_factory, "OTHER", cfg, "float32")
    reqs = prompts(cfg["vocab"], [90, 33, 2, 47, 64], seed=4)
    steps, peak = replay.cut_mixed(reqs, seed=7)
    os.makedirs(tmp_path / "out")
    rows = run_trace(d, steps, peak, str(tmp_path / "out"), cfg["vocab"])
    check(rows, expected(d, cfg, reqs), "float32", reqs)


def run_trace(model_dir, steps, max_tokens, out_dir, vocab):
    import subprocess
    import sys
    cmd = [sys.executable, os.path.join(replay.ROOT, "bin", "trace_run"), "--model", model_dir,
           "--dtype", "float32", "--out", out_dir, "--max-tokens", str(max_tokens)]
    p = subprocess.Popen(cmd, stdin=subprocess.PIPE, stdout=subprocess.PIPE, text=True)
    try:
        for s in steps:
            p.stdin.write(json.dumps(s) + "\n")
            p.stdin.flush()
            assert p.stdout.readline().strip() == f"done {s['step']}"
        p.stdin.close()
        assert p.wait(timeout=120) == 0
    finally:
        if p.poll() is None:
            p.kill()
    return replay.collect(steps, lambda i: np.fromfile(os.path.join(out_dir, f"{i}.f32"),
                                                       dtype="<f4").reshape(-1, vocab))


# ----------------------------------------------------------------------------- a key at a window's edge
def _edge_cuts(reqs, before, around):
    return (replay.cut_whole(reqs), replay.cut_tail_decode(reqs, tail=1),
            replay.cut_tail_decode(reqs, tail=around + 3),
            replay.cut_portions(reqs, sizes=(max(1, before), 5, 2, 3, max(2, around), 7)))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window, page", [(37, 16), (16, 16), (48, 8), (2, 16), (5, 4), (64, 16),
                                          (100, 32)])
def test_a_key_just_inside_and_just_outside_the_window(tmp_path_factory, window, page, dtype):
    """The probing token asks for the target token alone.  The target sits ``window - 1`` tokens
    before the probe (the last key the window keeps) or ``window`` before it (the first one it has
    lost); the probe is a row of the whole prompt, of a later portion, and decoded alone, with the
    target decoded as well or part of the prompt."""
    cfg, tensors = tl.edge_attention_model(window)
    d = folder(tmp_path_factory, f"EDGE{window}", cfg, dtype, tensors)
    W = stored(d)
    rng = random.Random(window)
    probe_at = 2 * window + 70
    answers = {}
    for place, target_at in (("in", probe_at - window + 1), ("out", probe_at - window)):
        toks = [rng.randrange(3, cfg["vocab"]) for _ in range(probe_at + 1)]
        toks[target_at], toks[probe_at] = tl.TARGET, tl.PROBE
        want = plain.forward(cfg, W, toks).numpy()
        answers[place] = want[probe_at]
        reqs = {"e": toks}
        for cut in _edge_cuts(reqs, target_at - 2, window):
            runner = make_runner(d, dtype, len(toks) + 64, page_size=page)
            rows = replay.run_in_process(runner, cut)
            err = rel(rows[("e", probe_at)], want[probe_at])
            assert err <= (2e-4 if dtype == "float32" else 0.05), (place, err)
    # the two places give different answers: the probe reads the target's value or it does not
    dlt = answers["in"] - answers["out"]
    assert np.sqrt((dlt ** 2).mean()) > 0.2 * np.sqrt((answers["in"] ** 2).mean())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("target_at, page", [(0, 16), (15, 16), (16, 16), (17, 16), (255, 8),
                                             (256, 32), (3, 4)])
def test_attention_without_a_window_finds_a_far_key_among_hundreds(tmp_path_factory, target_at, page,
                                                                   dtype):
    """The probe, 600 tokens on, asks for a target at the sequence's start, at a page's last and
    first place, and the answer differs from the one without the target."""
    cfg, tensors = tl.edge_attention_model(0, vdim=32)
    d = folder(tmp_path_factory, "EDGE_FAR", cfg, dtype, tensors)
    W = stored(d)
    rng = random.Random(target_at)
    probe_at = 600
    toks = [rng.randrange(3, cfg["vocab"]) for _ in range(probe_at + 1)]
    toks[probe_at] = tl.PROBE
    without = plain.forward(cfg, W, toks).numpy()[probe_at]
    toks[target_at] = tl.TARGET
    want = plain.forward(cfg, W, toks).numpy()
    assert rel(without.astype(np.float32), want[probe_at]) > 0.2
    reqs = {"e": toks}
    for cut in _edge_cuts(reqs, target_at + 1, 30):
        runner = make_runner(d, dtype, len(toks) + 64, page_size=page)
        rows = replay.run_in_process(runner, cut)
        err = rel(rows[("e", probe_at)], want[probe_at])
        assert err <= (2e-4 if dtype == "float32" else 0.05), err


# ----------------------------------------------------------------------------- generation
@pytest.mark.parametrize("pages", [None, 14])
def test_greedy_generation_through_the_entry_point(tmp_path_factory, pages):
    from ginfer_b200.engine.llm import Engine
    from ginfer_b200.sampling import SamplingParams
    cfg = tl.MIXED
    d = folder(tmp_path_factory, "MIXED", cfg, "float32")
    reqs = prompts(cfg["vocab"], [40, 9, 75, 1, 23], seed=6)
    eng = Engine(d, dtype="float32", max_num_seqs=3, max_num_batched_tokens=64, max_seq_len=128,
                 num_kvcache_blocks=pages, kvcache_block_size=8)
    outs = eng.generate(list(reqs.values()), SamplingParams(temperature=0.0, max_tokens=10,
                                                             ignore_eos=True))
    W = stored(d)
    for toks, out in zip(reqs.values(), outs):
        assert len(out) == 10
        seq = list(toks)
        for t in out:
            logits = plain.forward(cfg, W, seq)[-1]
            if int(torch.argmax(logits)) != t:           # only a close call may differ
                assert float(logits.max() - logits[t]) < 1e-3 * float(logits.abs().max()), (seq, t)
            seq.append(t)
    if pages is not None:
        eng.runner.cache.check()


def test_generation_from_the_command_line(tmp_path_factory, tmp_path):
    import subprocess
    import sys
    cfg = tl.OTHER
    d = folder(tmp_path_factory, "OTHER", cfg, "float32")
    reqs = prompts(cfg["vocab"], [6, 11], seed=10)
    f = tmp_path / "prompts.txt"
    f.write_text("\n".join(json.dumps(t) for t in reqs.values()) + "\n")
    r = subprocess.run([sys.executable, os.path.join(replay.ROOT, "bin", "ginfer_generate"),
                        "--model-path", d, "--dtype", "float32", "--prompt-ids", str(f),
                        "--max-tokens", "5", "--ignore-eos", "--max-num-seqs", "2",
                        "--max-seq-len", "64", "--num-kvcache-blocks", "8"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(x) for x in r.stdout.strip().splitlines()]
    W = stored(d)
    for toks, line in zip(reqs.values(), lines):
        seq = list(toks)
        assert len(line["output_ids"]) == 5
        for t in line["output_ids"]:
            logits = plain.forward(cfg, W, seq)[-1]
            if int(torch.argmax(logits)) != t:
                assert float(logits.max() - logits[t]) < 1e-3 * float(logits.abs().max())
            seq.append(t)


# ----------------------------------------------------------------------------- kernels alone
class _Ctx:
    extras: dict = {}


def packed(q_lens, slots, starts=None):
    """A step's facts for kernels that read them: portions of ``q_lens`` rows of the requests in
    ``slots``."""
    ctx = _Ctx()
    ctx.extras = {}
    i32 = dict(dtype=torch.int32, device="cuda")
    ctx.num_seqs, ctx.num_tokens, ctx.max_q_len = len(q_lens), sum(q_lens), max(q_lens)
    ctx.q_lens_host, ctx.decode_only = list(q_lens), max(q_lens) == 1
    ctx.cu_seqlens_q = torch.tensor([0] + list(np.cumsum(q_lens)), **i32)
    ctx.seq_of_token = torch.tensor([b for b, n in enumerate(q_lens) for _ in range(n)], **i32)
    ctx.slot_ids = torch.tensor(slots, **i32)
    return ctx


def close(got, want, tol):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape
    assert torch.allclose(got, want, atol=tol, rtol=tol), float((got - want).abs().max())


@pytest.mark.parametrize("act", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H", [48, 50, 256, 520, 1030, 2048, 4104, 8192])
def test_sublayer_end_and_the_shifted_norm_in_one_kernel(H, act):
    """Three requests in slots 4, 1, 2 over several steps (portions of every kind: a single token, one
    that ends inside a block's rows, one that spans blocks, all single tokens) against one pass over
    whole sequences; other slots keep their rows."""
    from ginfer_b200.ops import shift
    g = torch.Generator().manual_seed(H)
    lens, slots = [41, 23, 30], [4, 1, 2]
    steps = [[1, 2, 17], [19, 1, 1], [1, 1, 1], [3, 7, 2], [1, 1, 8], [16, 11, 1]]
    assert [sum(s[b] for s in steps) for b in range(3)] == lens
    X = [torch.randn(n, H, generator=g) for n in lens]
    ydt = act
    Y = [(torch.randn(n, H, generator=g) * 3).to(ydt) for n in lens]
    gb, gn, w = (torch.rand(H, generator=g) + 0.5 for _ in range(3))
    for with_y in (True, False):
        V, N = [], []
        for x, y in zip(X, Y):
            v = x.double()
            if with_y:
                v = v + plain.rms_norm(y.double(), 1e-3, gb.double())
            V.append(v)
            N.append(plain.rms_norm(v, 1e-5, gn.double()))
        want = [plain.token_shift(n, w.double()) for n in N]
        state = torch.zeros(6, H, device="cuda")
        state[0] = state[3] = 7.0
        at = [0, 0, 0]
        tol = 2e-5 if act == torch.float32 else 3e-2
        for q_lens in steps:
            ctx = packed(q_lens, slots)
            rows = [slice(a, a + n) for a, n in zip(at, q_lens)]
            x = torch.cat([t[r] for t, r in zip(X, rows)]).cuda()
            y = torch.cat([t[r] for t, r in zip(Y, rows)]).cuda()
            kw = dict(y=y, gamma_b=gb.cuda(), eps_b=1e-3) if with_y else {}
            v, h = shift.norm_shift(x, act, gn.cuda(), 1e-5, w.cuda(), state, ctx, **kw)
            assert h.dtype == act and (with_y or v is x)
            close(v, torch.cat([t[r] for t, r in zip(V, rows)]), 2e-5)
            close(h, torch.cat([t[r] for t, r in zip(want, rows)]), tol)
            at = [a + n for a, n in zip(at, q_lens)]
            for b, s in enumerate(slots):                    # never rounded to 16 bits
                close(state[s], N[b][at[b] - 1], 2e-5)
        assert float((state[[0, 3]] - 7.0).abs().max()) == 0.0 and float(state[5].abs().max()) == 0.0


def test_shifted_norm_of_a_long_portion_and_a_wide_output_type_of_y():
    from ginfer_b200.ops import shift
    g = torch.Generator().manual_seed(1)
    for H in (2048, 324):
        T = 300
        x, y = torch.randn(T, H, generator=g), torch.randn(T, H, generator=g)
        gb, gn, w = (torch.rand(H, generator=g) + 0.5 for _ in range(3))
        state = torch.randn(3, H, generator=g).cuda()
        first = state[2].double().cpu()
        v, h = shift.norm_shift(x.cuda(), torch.bfloat16, gn.cuda(), 1e-5, w.cuda(), state,
                                packed([T], [2]), y=y.cuda(), gamma_b=gb.cuda(), eps_b=1e-3)
        n = plain.rms_norm(x.double() + plain.rms_norm(y.double(), 1e-3, gb.double()), 1e-5, gn.double())
        before = torch.cat([first[None], n[:-1]])
        close(h, n + (before - n) * w.double(), 3e-2)
        close(state[2], n[-1], 2e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh, nkv, D, Vd, P, dims, yarn", [
    (4, 2, 16, 12, None, 8, True), (3, 1, 24, 28, None, 24, True), (6, 2, 56, 44, 64, 28, True),
    (5, 5, 14, 9, None, 6, False), (2, 1, 96, 80, 128, 48, True), (3, 3, 33, 8, None, 0, False),
    (16, 4, 128, 128, None, 64, True), (2, 2, 192, 160, None, 100, True), (4, 1, 40, 64, 64, 40, True)])
def test_rotation_then_norm_of_heads_and_the_cache_write(dtype, nh, nkv, D, Vd, P, dims, yarn):
    """Positions far apart, heads with and without zero padding (``P``), every share of rotated
    channels, values of another size, sizes that take four channels an access and sizes that do not."""
    from ginfer_b200.ops import prenorm
    rot = {"dims": dims, "base": 700.0, "scaling": tl.YARN if yarn else None}
    freqs, mult = plain.yarn_frequencies(rot)
    g = torch.Generator().manual_seed(D)
    T, slots = 13, 40
    kd, vd = P or D, P or Vd
    ld = (nh + nkv) * kd + nkv * vd
    ld += -ld % 8
    qkv = torch.zeros(T, ld)
    qkv[:, :nh * kd].view(T, nh, kd)[..., :D] = torch.randn(T, nh, D, generator=g) * 2
    k_off, v_off = nh * kd, (nh + nkv) * kd
    qkv[:, k_off:v_off].view(T, nkv, kd)[..., :D] = torch.randn(T, nkv, D, generator=g)
    qkv[:, v_off:v_off + nkv * vd].view(T, nkv, vd)[..., :Vd] = torch.randn(T, nkv, Vd, generator=g)
    qkv = qkv.to(dtype)
    pos = torch.tensor([0, 1, 2, 15, 16, 17, 63, 64, 255, 256, 777, 1023, 4095][:T]).int()
    slot = torch.randperm(slots, generator=g)[:T].int()
    kp = torch.zeros(slots, 1, nkv, kd, dtype=dtype).cuda()
    vp = torch.zeros(slots, 1, nkv, vd, dtype=dtype).cuda()
    dev = qkv.clone().cuda()
    prenorm.qk_rope_norm(dev, nh, nkv, kd, vd, D, k_off, v_off, 1e-5,
                         freqs.float().cuda() if dims else None, mult, pos.cuda(), slot.cuda(), kp, vp)
    x = qkv.double()

    def turned(t):
        full = torch.zeros(4096, t.shape[1], D, dtype=F64)
        full[pos.long()] = t
        return plain.rms_norm(plain.rotate(full, freqs, mult)[pos.long()], 1e-5)
    q = turned(x[:, :k_off].reshape(T, nh, kd)[..., :D])
    k = turned(x[:, k_off:v_off].reshape(T, nkv, kd)[..., :D])
    # (fp32 angles of positions in the thousands: 1e-4)
    tol = 5e-4 if dtype == torch.float32 else 3e-2
    got_q = dev[:, :k_off].cpu().reshape(T, nh, kd)
    got_k = kp[slot.long(), 0].cpu()
    close(got_q[..., :D], q, tol)
    close(got_k[..., :D], k, tol)
    assert float(got_q[..., D:].abs().sum()) == 0.0 and float(got_k[..., D:].abs().sum()) == 0.0
    assert torch.equal(vp[slot.long(), 0].cpu(), qkv[:, v_off:v_off + nkv * vd].reshape(T, nkv, vd))
    assert torch.equal(dev[:, k_off:].cpu(), qkv[:, k_off:])           # k and v stay as projected
    kp2 = torch.zeros_like(kp)
    dev2 = qkv.clone().cuda()
    prenorm.qk_rope_norm(dev2, nh, nkv, kd, vd, D, k_off, v_off, 1e-5,
                         freqs.float().cuda() if dims else None, mult, pos.cuda(), None, kp2, vp)
    assert float(kp2.abs().max()) == 0.0 and torch.equal(dev2, dev)


def _paged_kv(keys, page, nkv, D, Vd, dtype, g):
    npages = -(-keys // page)
    order = torch.randperm(npages + 3, generator=g)[:npages]
    k = torch.randn(keys, nkv, D, generator=g).to(dtype)
    v = torch.randn(keys, nkv, Vd, generator=g).to(dtype)
    kp = torch.zeros(npages + 3, page, nkv, D, dtype=dtype)
    vp = torch.zeros(npages + 3, page, nkv, Vd, dtype=dtype)
    for j in range(keys):
        kp[order[j // page], j % page] = k[j]
        vp[order[j // page], j % page] = v[j]
    if D == Vd:
        return k.double(), v.double(), torch.stack([kp, vp]).cuda(), order
    return k.double(), v.double(), (kp.cuda(), vp.cuda()), order


def _sink_reference(q, k, v, p, nh, nkv, scale, window, sink):
    lo = max(0, p - window + 1) if window > 0 else 0
    out = []
    for n in range(nh):
        s = (k[lo:p + 1, n // (nh // nkv)] @ q[n]) * scale
        w = torch.softmax(torch.cat([s, torch.tensor([sink], dtype=F64)]), 0)[:-1]
        out.append(w @ v[lo:p + 1, n // (nh // nkv)])
    return torch.stack(out)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh, nkv, D, Vd, window, sink, gain", [
    (4, 2, 64, 64, 100, 0.0, 1.0), (2, 2, 64, 64, 5, 0.0, 0.3), (16, 4, 128, 128, 0, 4.0, 1.0),
    (3, 1, 16, 16, 37, 0.0, 1.0), (6, 2, 24, 40, 19, 0.0, 1.0), (20, 1, 64, 64, 70, -2.0, 0.5),
    (4, 2, 48, 48, 3, 1.5, 1.0), (2, 1, 192, 192, 72, 0.0, 1.0), (4, 2, 64, 64, 1, 0.0, 30.0),
    (4, 2, 128, 128, 33, 90.0, 30.0)])
def test_attention_with_a_sink(dtype, nh, nkv, D, Vd, window, sink, gain):
    """The step's queries over a paged cache in shuffled pages with a sink in the denominator: every
    row of a prompt (tcgen05 from 64 rows in bfloat16 where the head size allows, ``mma.sync`` below;
    fp32 arithmetic elsewhere), single decoded rows of several requests, and single rows in front of
    a portion; flat scores over few keys (the sink's share is large), scores far above and below the
    sink, rows whose scores are all very negative."""
    from ginfer_b200 import ops
    g = torch.Generator().manual_seed(D + window)
    keys, page = 200, 8
    k, v, pages, order = _paged_kv(keys, page, nkv, D, Vd, dtype, g)
    q = (torch.randn(keys, nh, D, generator=g) * gain).to(dtype)
    scale = D ** -0.5
    table1 = order.int().cuda()[None, :]
    tol = 1e-4 if dtype == torch.float32 else 3e-2
    biggest = 0.0

    def run(rows_of, what):
        nonlocal biggest
        B, rows = len(rows_of), [p for r in rows_of for p in r]
        ctx = packed([len(r) for r in rows_of], list(range(B)))
        ctx.max_kv_len = max(r[-1] + 1 for r in rows_of)
        ctx.positions = torch.tensor(rows, dtype=torch.int32, device="cuda")
        ctx.kv_lens = torch.tensor([r[-1] + 1 for r in rows_of], dtype=torch.int32, device="cuda")
        kw = {} if D == Vd else {"vd": Vd}
        args = (q[rows].reshape(len(rows), nh * D).cuda().contiguous(), pages,
                table1.expand(B, -1).contiguous(), ctx, nh, nkv, D, scale, window, page)
        out = ops.paged_attention(*args, sink=sink, **kw).double().cpu().reshape(len(rows), nh, Vd)
        bare = ops.paged_attention(*args, **kw).double().cpu().reshape(len(rows), nh, Vd)
        for i, p in enumerate(rows):
            want = _sink_reference(q[p].double(), k, v, p, nh, nkv, scale, window, sink)
            assert torch.allclose(out[i], want, atol=tol, rtol=tol), (p, what)
            biggest = max(biggest, float((bare[i] - want).abs().max()))
    run([list(range(keys))], "prompt")                                   # a whole prompt
    run([list(range(130, keys))], "portion")                             # a later portion
    run([list(range(150, keys))], "short portion")                       # under the tcgen05 kernel's rows
    run([[keys - 1], [5], [window if window else 63], [0], [77]], "decode")
    run([[keys - 1], [40], list(range(90, 175))], "mixed")               # single rows, then a portion
    assert biggest > 3 * tol                                             # without the sink it shows


@pytest.mark.parametrize("B, keys, kw", [
    (1, 9000, dict(splits=8, parts=4)), (2, 700, dict(splits=1, parts=3)), (3, 900, dict(splits=4)),
    (2, 1500, dict(splits=16)), (2, 800, dict(splits=1)), (2, 800, dict(splits=5, use_tma=False)),
    (2, 800, dict(splits=8, use_tma=False)), (2, 800, dict(splits=16, use_tma=False)),
    (2, 300, dict(splits=1, use_tma=False)), (2, 800, dict(splits=4, through_scratch=True))])
def test_every_merge_of_split_decode_attention_counts_the_sink_once(B, keys, kw):
    from ginfer_b200.ops import attention_bf16
    g = torch.Generator().manual_seed(keys)
    nh, nkv, D, page = 6, 2, 64, 16
    k, v, pages, order = _paged_kv(keys, page, nkv, D, D, torch.bfloat16, g)
    q = (torch.randn(B, nh, D, generator=g) * 0.2).to(torch.bfloat16)
    pos = [keys - 1 - 37 * b for b in range(B)]
    sink = 8.0
    out = attention_bf16.decode(
        q.reshape(B, nh * D).cuda(), pages, order.int().cuda()[None].expand(B, -1).contiguous(), None,
        torch.tensor(pos, dtype=torch.int32, device="cuda"), B, nh, nkv, D, D ** -0.5, 0, page,
        sink=sink, **kw).double().cpu().reshape(B, nh, D)
    for b in range(B):
        want = _sink_reference(q[b].double(), k, v, pos[b], nh, nkv, D ** -0.5, 0, sink)
        err = float((out[b] - want).abs().max())
        assert err < 0.02 * float(want.abs().max()) + 1e-4, (b, err)


@pytest.mark.parametrize("M", [1, 8, 16, 33, 64, 100, 700])
def test_xielu_in_the_products_epilogue_and_in_place(M):
    """From the tcgen05 kernel (direct tiles and K splits, by the token count), from the library
    product with the kernel behind it, and in 32-bit; both sides of zero and zero itself."""
    from ginfer_b200 import ops
    from ginfer_b200.ops import gemm_bf16
    g = torch.Generator(device="cuda").manual_seed(M)
    a, b = 0.71, 1.9

    def act(z):
        return torch.where(z > 0, a * z * z, b * (torch.expm1(torch.clamp(z, max=0.0))
                                                  - torch.clamp(z, max=0.0))) + z / 2
    for K, N in ((192, 328), (4096, 136), (64, 1000)):
        x = torch.randn(M, K, generator=g, device="cuda").to(torch.bfloat16)
        w = (torch.randn(N, K, generator=g, device="cuda") * K ** -0.5 * 2).to(torch.bfloat16)
        w[:5] = 0
        bias = torch.randn(N, generator=g, device="cuda")
        bias[:3] = 0
        for bb in (bias, None):
            want = act(x.double() @ w.double().T + (bb.double() if bb is not None else 0))
            for out in (torch.bfloat16, torch.float32):
                y = ops.Linear(w, bb, out_dtype=out, activation="xielu", act_consts=(a, b))(x)
                assert y.dtype == out and y.shape == (M, N)
                tol = 0.02 if out == torch.bfloat16 else 2e-3
                assert float((y.double() - want).abs().max()) <= tol * float(want.abs().max())
                assert float(y[:, :3].abs().max()) == 0.0
            y32 = ops.Linear(w.float(), bb, activation="xielu", act_consts=(a, b))(x.float())
            assert torch.allclose(y32.double(), want, atol=1e-4, rtol=1e-4)
    gemm_bf16.check_errors("cuda:0")
    z = torch.tensor([-90.0, -3.0, -1e-3, -1e-6, 0.0, 1e-6, 0.4, 20.0], device="cuda")
    assert torch.allclose(ops.activation_(z.clone(), "xielu", a, b).double(), act(z.double()),
                          atol=1e-9, rtol=1e-5)


def _delta_case(G, H, D, Vd, taps, T, g):
    ch = 2 * G * D + H * Vd
    b_off = ch + H * Vd + H
    ld = b_off + H
    ld += -ld % 8
    p = torch.randn(T, ld, generator=g)
    conv = torch.randn(ch, taps, generator=g) * 0.7
    return p, conv, torch.randn(H, generator=g) * 0.5, torch.linspace(-3.0, 0.5, H), ch, b_off - H, b_off


def _delta_want(p, conv, bias, A, ch, a_off, b_off, G, H, D, Vd):
    p = p.double()
    y = plain.silu(plain.causal_conv(p[:, :ch], conv.double()))
    T = p.shape[0]
    q = plain.unit(y[:, :G * D].reshape(T, G, D)) * D ** -0.5
    k = plain.unit(y[:, G * D:2 * G * D].reshape(T, G, D))
    v = y[:, 2 * G * D:].reshape(T, H, Vd)
    g = plain.head_decay(p[:, a_off:a_off + H], A.double(), bias.double())
    beta = torch.sigmoid(p[:, b_off:b_off + H])
    o = torch.stack([plain.delta_rule(q[:, n // (H // G)], k[:, n // (H // G)], v[:, n], g[:, n],
                                      beta[:, n]) for n in range(H)], 1)
    return q, k, v, g, beta, o


@pytest.mark.parametrize("G, H, D, Vd, taps", [
    (2, 4, 8, 12, 4), (1, 3, 10, 9, 3), (2, 2, 128, 64, 4), (1, 2, 36, 200, 2), (3, 6, 7, 5, 5),
    (2, 6, 64, 32, 1), (1, 1, 256, 16, 3), (4, 4, 16, 128, 3), (1, 2, 12, 8, 6)])
def test_delta_rule_with_one_decay_a_head(G, H, D, Vd, taps):
    """Operands (convolution over portions and single tokens, unit vectors, decays, betas), the
    recurrence and the slots, for two requests under cuts of every kind; sizes that take four
    channels a lane and sizes that do not."""
    from ginfer_b200.ops import delta
    g = torch.Generator().manual_seed(D * taps)
    lens, slots = [90, 61], [2, 0]
    cases = [_delta_case(G, H, D, Vd, taps, n, g) for n in lens]
    _, conv, bias, A, ch, a_off, b_off = cases[0]
    wants = [_delta_want(c[0], conv, bias, A, ch, a_off, b_off, G, H, D, Vd) for c in cases]
    conv_off = H * D * Vd
    dev = [t.cuda() for t in (conv, bias, A)]
    for steps in ([[90, 61]], [[70, 1], [1, 1], [1, 40], [2, 2], [3, 17], [13, 0]],
                  [[1, 1]] * 6 + [[2, 3], [82, 52]]):
        state = torch.zeros(4, conv_off + (taps - 1) * ch, device="cuda")
        state[1] = state[3] = 5.0
        at = [0, 0]
        for q_lens in steps:
            ids = [b for b in range(2) if q_lens[b]]
            ctx = packed([q_lens[b] for b in ids], [slots[b] for b in ids])
            rows = [slice(at[b], at[b] + q_lens[b]) for b in ids]
            p = torch.cat([cases[b][0][r] for b, r in zip(ids, rows)]).cuda()
            q, k, v, gg, beta = delta.prepare_heads(p, a_off, b_off, dev[0], dev[1], dev[2], state, ctx,
                                                    H, G, D, Vd, taps, conv_off)
            o = delta.recurrence(q, k, v, gg, beta, state, ctx)
            for got, j, tol in ((q, 0, 1e-5), (k, 1, 1e-5), (v, 2, 1e-5), (gg, 3, 1e-5), (beta, 4, 1e-5),
                                (o, 5, 1e-4)):
                want = torch.cat([wants[b][j][r] for b, r in zip(ids, rows)])
                close(got, want, tol)
            at = [a + n for a, n in zip(at, q_lens)]
            for b in range(2):                       # the convolutions' last inputs
                for m in range(taps - 1):
                    i = at[b] - (taps - 1) + m
                    have = state[slots[b], conv_off + m * ch:conv_off + (m + 1) * ch].cpu()
                    assert torch.equal(have, cases[b][0][i, :ch] if i >= 0 else torch.zeros(ch)), (b, m)
        assert at == lens
        assert float((state[[1, 3]] - 5.0).abs().max()) == 0.0


@pytest.mark.parametrize("D, Vd, per", [(16, 24, 1), (20, 8, 3), (64, 40, 2), (128, 128, 1), (200, 12, 2)])
def test_eight_tokens_at_a_time_agree_with_one_by_one(D, Vd, per):
    """The recurrence of long portions against the token-by-token kernel and the plain one, from a
    state that is not zero, over portions of 16 to 100 tokens beside single ones (ends inside a
    chunk); keys that repeat with a step size of one (every token undoes the last one's write),
    decays of exactly one and decays that forget at once."""
    from ginfer_b200.ops import delta
    g0 = torch.Generator().manual_seed(D)
    G, H = 2, 2 * per
    q_lens, slots = [100, 1, 16, 23, 40], [3, 0, 5, 1, 2]
    T = sum(q_lens)
    k = plain.unit(torch.randn(T, G, D, generator=g0))
    k[101:117, 0] = k[101, 0]                               # one key for a whole portion
    q = plain.unit(torch.randn(T, G, D, generator=g0)) * D ** -0.5
    v = torch.randn(T, H, Vd, generator=g0)
    beta = torch.rand(T, H, generator=g0)
    beta[101:117] = 1.0
    gg = torch.rand(T, H, generator=g0) ** 0.2
    gg[0:40, 0] = 1.0
    gg[50::7, -1] = 1e-30
    S0 = torch.randn(6, H * D * Vd, generator=g0)
    args = [t.float().cuda().contiguous() for t in (q, k, v, gg, beta)]
    ctx = packed(q_lens, slots)
    outs = []
    for min_tokens in (16, 1 << 30):
        old, delta.CHUNKED_MIN_TOKENS = delta.CHUNKED_MIN_TOKENS, min_tokens
        try:
            state = S0.cuda()
            outs.append((delta.recurrence(*args, state, ctx).cpu(), state.cpu()))
        finally:
            delta.CHUNKED_MIN_TOKENS = old
    (o8, s8), (o1, s1) = outs
    scale = float(o1.abs().max())
    assert float((o8 - o1).abs().max()) <= 2e-5 * scale and not torch.equal(o8, o1)
    assert float((s8 - s1).abs().max()) <= 2e-5 * float(s1.abs().max())
    assert torch.equal(s8[4], S0[4])
    at = 0
    for n, slot in zip(q_lens, slots):
        S = S0[slot].double().view(H, D, Vd).clone()
        for t in range(at, at + n):
            for h in range(H):
                kk, qq = k[t, h // per].double(), q[t, h // per].double()
                S[h] = float(gg[t, h]) * S[h]
                u = float(beta[t, h]) * (v[t, h].double() - S[h].T @ kk)
                S[h] = S[h] + torch.outer(kk, u)
                want = S[h].T @ qq
                assert float((o8[t, h].double() - want).abs().max()) <= 5e-5 * scale, (t, h)
        assert float((s8[slot].double() - S.view(-1)).abs().max()) <= 5e-5 * float(S.abs().max())
        at += n


def test_delta_operands_of_a_long_prompt_among_others():
    """Enough tokens that a warp walks over runs of them: runs that start inside a portion, at its
    start, and that cross from one request to the next."""
    from ginfer_b200.ops import delta
    g = torch.Generator().manual_seed(9)
    G, H, D, Vd, taps = 2, 4, 32, 48, 4
    lens, slots = [301, 3, 130], [1, 0, 2]
    cases = [_delta_case(G, H, D, Vd, taps, n, g) for n in lens]
    _, conv, bias, A, ch, a_off, b_off = cases[0]
    state = torch.zeros(3, H * D * Vd + (taps - 1) * ch, device="cuda")
    ctx = packed(lens, slots)
    p = torch.cat([c[0] for c in cases]).cuda()
    got = delta.prepare_heads(p, a_off, b_off, conv.cuda(), bias.cuda(), A.cuda(), state, ctx, H, G, D,
                              Vd, taps, H * D * Vd)
    wants = [_delta_want(c[0], conv, bias, A, ch, a_off, b_off, G, H, D, Vd) for c in cases]
    for j in range(5):
        close(got[j], torch.cat([w[j] for w in wants]), 1e-5)


@pytest.mark.parametrize("D, Vd", [(16, 8), (64, 64), (128, 128), (100, 30)])
def test_a_far_write_is_read_back_as_the_decay_left_it(D, Vd):
    """A value written at the first token under a key that no later token uses is read back 300
    tokens later, faded by the product of the decays, in one portion, token by token and in uneven
    portions, also in a large batch (the other width of the recurrence)."""
    from ginfer_b200.ops import delta
    T = 300
    g0 = torch.Generator().manual_seed(D)
    for H, B in ((2, 1), (4, 40)):
        k = torch.zeros(T, 1, D)
        k[0, 0, 0] = 1.0
        for t in range(1, T):
            k[t, 0, 1 + t % (D - 1)] = 1.0
        q = torch.zeros(T, 1, D)
        q[:, :, 0] = 1.0
        v = torch.randn(T, H, Vd, generator=g0)
        gg = 1.0 - torch.rand(T, H, generator=g0) * 0.01
        beta = torch.full((T, H), 0.8)
        want = 0.8 * v[0].double() * gg[1:].double().prod(0)[:, None]
        order = torch.randperm(B + 2, generator=g0)[:B].tolist()
        for cut in ([T], [7, 2, 100, 1, 190]) + (([1] * T,) if B == 1 else ()):
            state = torch.zeros(B + 2, H * D * Vd, device="cuda")
            at, o = 0, None
            for n in cut:
                sl = slice(at, at + n)
                rep = [t[sl].repeat(B, *([1] * (t.dim() - 1))).cuda().contiguous()
                       for t in (q, k, v, gg, beta)]
                o = delta.recurrence(*rep, state, packed([n] * B, order))
                at += n
            got = o.view(B, -1, H, Vd)[:, -1].double().cpu()
            assert torch.allclose(got, want[None].expand(B, -1, -1), atol=1e-5), (B, cut[:3])
