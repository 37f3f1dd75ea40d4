"""Daburax on the device against the plain implementation (``plain_daburax``): every mechanism alone,
whole prompts against token-by-token decoding, portions down to two tokens, batches of unequal requests,
pages and slots used again, a far key that stands out at page borders, in prompts and decoded, the first
tokens of a sequence, long decoding through CUDA graphs, other sizes, greedy generation through the entry
point, and the kernels alone."""
import json
import os
import random

import numpy as np
import pytest
import torch

import plain_daburax as plain
import replay
import tiny_daburax as td

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64
_folders: dict = {}
_expected: dict = {}


def folder(tmp_path_factory, name, cfg, dtype, tensors=None):
    key = (name, dtype)
    if key not in _folders:
        path = str(tmp_path_factory.mktemp(f"daburax_{name}_{dtype}"))
        _folders[key] = td.write_folder(path, cfg, seed=len(name), storage=DTYPES[dtype],
                                        tensors=tensors)
    return _folders[key]


def stored(model_dir):
    """The folder's tensors as float64 (what the file holds, not what was drawn)."""
    from ginfer_b200.weights.safetensors_io import open_model_tensors
    return {n: f.get(k).double() for n, (f, k) in open_model_tensors(model_dir).items()}


def prompts(vocab, lengths, seed=0):
    rng = random.Random(seed)
    return {f"r{i}": [rng.randrange(vocab) for _ in range(n)] for i, n in enumerate(lengths)}


def bf16(x):
    return x.float().bfloat16().double()


def expected(model_dir, cfg, requests, dtype="float32", **kw):
    """The plain logits; for bfloat16 with the activations rounded where the engine stores them."""
    out = {}
    W = None
    for rid, toks in requests.items():
        key = (model_dir, tuple(toks), dtype, tuple(sorted(kw.items())))
        if key not in _expected:
            W = W or stored(model_dir)
            rnd = bf16 if dtype == "bfloat16" else plain.same
            _expected[key] = plain.forward(cfg, W, toks, rnd=rnd, **kw).numpy()
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


# float32: differences of summation order.  bfloat16: a router's close call may fall the other way and
# peaked attention amplifies the format's rounding, so single rows may be off (at most one in fifteen)
# while the middle row is close; a misplaced page, a lost state or a token that is not seen puts most
# rows near one.
LIMIT = {"float32": (1e-4, 1e-5), "bfloat16": (0.15, 0.04)}


def check(rows, want, dtype, requests):
    assert len(rows) == sum(len(t) for t in requests.values()), "a logits row is missing"
    errs = {key: rel(row, want[key[0]][key[1]]) for key, row in sorted(rows.items())}
    where = max(errs, key=errs.get)
    if dtype == "bfloat16":
        over = sum(not e <= LIMIT[dtype][0] for e in errs.values())
        assert over <= max(1, len(errs) // 15), \
            f"{over} of {len(errs)} rows are off; worst {where}: {errs[where]:.3e}"
    else:
        assert errs[where] <= LIMIT[dtype][0], f"worst row {where}: relative error {errs[where]:.3e}"
    middle = float(np.median(list(errs.values())))
    assert middle <= LIMIT[dtype][1], f"median relative error {middle:.3e}"


# ----------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["RETENTION_ONLY", "PARALLEL_ONLY", "MOE_FF", "BIGRAM"])
def test_each_mechanism_alone(tmp_path_factory, name, dtype):
    cfg = getattr(td, name)
    d = folder(tmp_path_factory, name, cfg, dtype)
    reqs = prompts(cfg["vocab"], [70, 3, 1])
    want = expected(d, cfg, reqs, dtype)
    for steps in (replay.cut_whole(reqs), replay.cut_portions(reqs)):
        rows = replay.run_in_process(make_runner(d, dtype, replay.peak_tokens(steps)), steps)
        check(rows, want, dtype, reqs)


@pytest.mark.parametrize("without", [
    "bigram", "rot", "scaling", "decay", "head_norm", "gate", "bias", "sink", "cap", "input_gate",
    "forget_gate", "left", "right", "correction", "groups", "identity", "shared", "shared_gate", "mix",
    "mix_transposed"])
def test_the_oracle_without_a_mechanism_is_far_from_the_oracle(tmp_path_factory, without):
    """Passing the comparisons means the mechanism was computed: leaving it out moves the logits by
    much more than any limit."""
    cfg = td.MIXED
    d = folder(tmp_path_factory, "MIXED", cfg, "float32")
    reqs = prompts(cfg["vocab"], [60], seed=11)
    full = expected(d, cfg, reqs)["r0"]
    less = expected(d, cfg, reqs, without=(without,))["r0"]
    assert np.mean([rel(less[p].astype(np.float32), full[p]) for p in range(20, 60)]) > 0.01


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
    cfg = getattr(td, name)
    d = folder(tmp_path_factory, name, cfg, dtype)
    reqs = prompts(cfg["vocab"], LENGTHS, seed=1)
    want = expected(d, cfg, reqs, dtype)
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


@pytest.mark.parametrize("name", ["MIXED", "OTHER", "BIGRAM"])
def test_the_first_tokens_of_a_sequence(tmp_path_factory, name):
    """Positions 0, 1, 2: no token before the first one, empty states, a running maximum that starts at
    zero, one key beside the sink; as a prompt of their own, as the start of a longer one, one by one,
    and behind another request that left its slot and pages."""
    cfg = getattr(td, name)
    d = folder(tmp_path_factory, name, cfg, "float32")
    reqs = prompts(cfg["vocab"], [50, 3, 2, 1], seed=21)
    want = expected(d, cfg, reqs)
    for steps in (replay.cut_whole(reqs), replay.cut_tail_decode(reqs, tail=60),
                  replay.cut_portions(reqs, sizes=(1, 2, 1, 1, 40))):
        runner = make_runner(d, "float32", 64, max_live=1)
        rows = replay.run_in_process(runner, steps)
        check(rows, want, "float32", reqs)


@pytest.mark.parametrize("name, dtype", [("MIXED", "float32"), ("WIDE", "bfloat16")])
def test_long_decoding_through_graphs(tmp_path_factory, name, dtype):
    cfg = getattr(td, name)
    d = folder(tmp_path_factory, name, cfg, dtype)
    reqs = prompts(cfg["vocab"], [230], seed=2)
    steps = replay.cut_tail_decode(reqs, tail=200)       # 30 in one step, then 200 single tokens
    runner = make_runner(d, dtype, replay.peak_tokens(steps), eager=False)
    check(replay.run_in_process(runner, steps), expected(d, cfg, reqs, dtype), dtype, reqs)
    assert runner.graph_launches > 0


def test_decoded_batches_of_many_sizes_through_graphs(tmp_path_factory):
    """Ten requests decode together, fewer and fewer as they end, in batches whose graphs are padded
    with rows that belong to no request; slots and pages go to later requests."""
    cfg = td.MIXED
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
    cfg = getattr(td, name)
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
    check(rows, expected(d, cfg, reqs, "bfloat16"), "bfloat16", reqs)
    assert any(isinstance(k[0], str) for k in runner._graphs), "no portion step was captured"


def test_trace_program(tmp_path_factory, tmp_path):
    import subprocess
    import sys
    cfg = td.OTHER
    d = folder(tmp_path_factory, "OTHER", cfg, "float32")
    reqs = prompts(cfg["vocab"], [90, 33, 2, 47, 64], seed=4)
    steps, peak = replay.cut_mixed(reqs, seed=7)
    out = tmp_path / "out"
    os.makedirs(out)
    cmd = [sys.executable, os.path.join(replay.ROOT, "bin", "trace_run"), "--model", d,
           "--dtype", "float32", "--out", str(out), "--max-tokens", str(peak)]
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
    rows = replay.collect(steps, lambda i: np.fromfile(os.path.join(out, f"{i}.f32"),
                                                       dtype="<f4").reshape(-1, cfg["vocab"]))
    check(rows, expected(d, cfg, reqs), "float32", reqs)


# ----------------------------------------------------------------------------- a far token that stands out
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "memory", "retention"])
@pytest.mark.parametrize("target_at, page", [(0, 16), (15, 16), (16, 16), (17, 16), (255, 8), (256, 32),
                                             (3, 4)])
def test_a_far_key_among_hundreds(tmp_path_factory, kind, target_at, page, dtype):
    """The probe, 600 tokens on, asks for a target at the sequence's start, at a page's last and first
    place, and the answer differs from the one without the target; as a row of the whole prompt, of later
    portions, and decoded, with the target decoded as well."""
    cfg, tensors = td.probe_model(kind)
    d = folder(tmp_path_factory, f"PROBE_{kind}", cfg, dtype, tensors)
    W = stored(d)
    rng = random.Random(target_at)
    probe_at = 600
    toks = [rng.randrange(3, cfg["vocab"]) for _ in range(probe_at + 1)]
    toks[probe_at] = td.PROBE
    without = plain.forward(cfg, W, toks).numpy()[probe_at]
    toks[target_at] = td.TARGET
    want = plain.forward(cfg, W, toks).numpy()
    assert rel(without.astype(np.float32), want[probe_at]) > 0.2
    reqs = {"e": toks}
    for cut in (replay.cut_whole(reqs), replay.cut_tail_decode(reqs, tail=1),
                replay.cut_tail_decode(reqs, tail=40),
                replay.cut_portions(reqs, sizes=(max(1, target_at - 1), 5, 2, 3, 64, 7, 130))):
        runner = make_runner(d, dtype, len(toks) + 64, page_size=page)
        rows = replay.run_in_process(runner, cut)
        err = rel(rows[("e", probe_at)], want[probe_at])
        assert err <= (2e-4 if dtype == "float32" else 0.05), err


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("length", [1, 2, 17, 129, 300])
def test_a_large_sink_scales_the_attention(tmp_path_factory, length, dtype):
    """A sink as large as a hundred flat keys: a sequence's answer depends on its length through it."""
    cfg, tensors = td.probe_model("attention", sink=float(np.log(100.0)))
    # values with a part in common: what a token reads is the softmax's share of the keys times that
    tensors["l0.mix.left.v.b"] = torch.linspace(-3.0, 3.0, 24)
    tensors["l0.mix.left.o"] *= 0.1
    d = folder(tmp_path_factory, "PROBE_SINK", cfg, dtype, tensors)
    reqs = prompts(cfg["vocab"], [length], seed=length)
    W = stored(d)
    want = plain.forward(cfg, W, reqs["r0"]).numpy()
    bare = plain.forward(cfg, W, reqs["r0"], without=("sink",)).numpy()
    assert rel(bare[-1].astype(np.float32), want[-1]) > 0.05
    for steps in (replay.cut_whole(reqs), replay.cut_tail_decode(reqs, tail=3)):
        rows = replay.run_in_process(make_runner(d, dtype, 320), steps)
        assert rel(rows[("r0", length - 1)], want[-1]) <= (1e-4 if dtype == "float32" else 0.03)


# ----------------------------------------------------------------------------- generation
@pytest.mark.parametrize("pages", [None, 14])
def test_greedy_generation_through_the_entry_point(tmp_path_factory, pages):
    from ginfer_b200.engine.llm import Engine
    from ginfer_b200.sampling import SamplingParams
    cfg = td.MIXED
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
    cfg = td.OTHER
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
    pass


def packed(q_lens, slots, starts=None):
    """A step's facts for kernels that read them: portions of ``q_lens`` rows of the requests in
    ``slots`` that start at the positions ``starts``."""
    ctx = _Ctx()
    ctx.extras = {}
    i32 = dict(dtype=torch.int32, device="cuda")
    ctx.num_seqs, ctx.num_tokens, ctx.max_q_len = len(q_lens), sum(q_lens), max(q_lens)
    ctx.q_lens_host, ctx.decode_only = list(q_lens), max(q_lens) == 1
    ctx.cu_seqlens_q = torch.tensor([0] + list(np.cumsum(q_lens)), **i32)
    ctx.seq_of_token = torch.tensor([b for b, n in enumerate(q_lens) for _ in range(n)], **i32)
    ctx.slot_ids = torch.tensor(slots, **i32)
    starts = starts or [0] * len(q_lens)
    ctx.positions = torch.tensor([s + i for s, n in zip(starts, q_lens) for i in range(n)], **i32)
    return ctx


def close(got, want, tol):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape
    assert torch.allclose(got, want, atol=tol, rtol=tol), float((got - want).abs().max())


@pytest.mark.parametrize("act", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("S, W", [(1, 48), (2, 50), (3, 256), (4, 2048), (4, 520), (5, 4104), (8, 1028),
                                  (9, 128), (4, 8192)])
def test_a_sublayers_end_on_several_streams(S, W, act):
    """All forms: dense terms with constants and factors a token, pairs of which some have no row, with and
    without a norm behind, streams that are still one row, only reading at chosen rows, no old streams."""
    from ginfer_b200.ops import hyper
    g = torch.Generator().manual_seed(S * W)
    R, top, n_rows = 11, 3, 20

    def rnd(*shape):
        return torch.randn(*shape, generator=g)
    x, base = rnd(R, S, W), rnd(R, W)
    mix, ow, iw, gamma = rnd(S, S), rnd(S), rnd(S), 1.0 + 0.3 * rnd(W)
    a0, a1, w0, w1 = rnd(R, W), rnd(R, W).to(act), rnd(R), rnd(R)
    rows, pw = rnd(n_rows, W), rnd(R, top)
    pos = torch.randint(0, n_rows, (R * top,), generator=g).to(torch.int32)
    pos[::4] = -1
    dev = lambda t: t.cuda()                                                          # noqa: E731
    pairs = (dev(rows), dev(pos), dev(pw), top)
    picked = torch.where(pos.view(R, top, 1) >= 0, rows[pos.clamp(min=0).long()].view(R, top, W),
                         torch.zeros(())).double()
    py = (picked * pw.double()[..., None]).sum(1)
    forms = [
        (x, dict(terms=[(dev(a0), 0.7, None)]), 0.7 * a0.double()),
        (x, dict(terms=[(dev(a0), 0.7, dev(w0)), (dev(a1), -1.3, dev(w1))], pairs=pairs),
         0.7 * w0.double()[:, None] * a0.double() - 1.3 * w1.double()[:, None] * a1.double() + py),
        (x, dict(terms=[(dev(a1), 2.0, dev(w1))]), 2.0 * w1.double()[:, None] * a1.double()),
        (x, dict(pairs=pairs), py),
        (base[:, None, :].expand(-1, S, -1), dict(terms=[(dev(a0), 1.0, None)]), a0.double())]
    for xs, kw, y in forms:
        xd = dev(base)[:, None, :].expand(-1, S, -1) if xs.stride(1) == 0 else dev(xs)
        want = torch.einsum("st,rsw->rtw", mix.double(), xs.double()) + ow.double()[None, :, None] * y[:, None]
        u = torch.einsum("t,rtw->rw", iw.double(), want)
        wn = u / torch.sqrt((u * u).mean(-1, keepdim=True) + 1e-4) * gamma.double()
        xo, n = hyper.update(xd, S, act, mix=dev(mix), out_w=dev(ow), in_w=dev(iw), norm_weight=dev(gamma),
                             norm_eps=1e-4, **kw)
        close(xo, want, 2e-4)
        close(n, wn, 2e-4 if act == torch.float32 else 2e-2)
        xo2, none = hyper.update(xd, S, act, mix=dev(mix), out_w=dev(ow), **kw)
        assert none is None and torch.equal(xo, xo2)
    pick = torch.tensor([7, 0, 7, 10], dtype=torch.int32)
    u = torch.einsum("s,rsw->rw", iw.double(), x[pick.long()].double())
    wn = u / torch.sqrt((u * u).mean(-1, keepdim=True) + 1e-4) * gamma.double()
    close(hyper.read(dev(x), dev(iw), dev(gamma), 1e-4, act, rows=dev(pick)), wn,
          2e-4 if act == torch.float32 else 2e-2)
    xo, _ = hyper.update(None, S, act, out_w=dev(ow), terms=[(dev(a0), 1.5, None)], pairs=pairs)
    close(xo, ow.double()[None, :, None] * (1.5 * a0.double() + py)[:, None], 2e-4)


@pytest.mark.parametrize("H, act", [(50, torch.float32), (64, torch.bfloat16), (1030, torch.float32)])
def test_pair_embedding_and_its_state(H, act):
    """Three requests in slots 4, 1, 2 over several steps; other slots keep their token."""
    from ginfer_b200.ops import hyper
    g = torch.Generator().manual_seed(H)
    V, buckets, mp, mc = 91, 29, 1 << 33, 7            # (a multiplier over 32 bits)
    emb, table = torch.randn(V, H, generator=g).to(act), torch.randn(buckets + 1, H, generator=g).to(act)
    seqs = [torch.randint(0, V, (n,), generator=g).tolist() for n in (40, 23, 31)]
    want = [emb.double()[torch.tensor(s)] * 1.5 +
            table.double()[torch.tensor(plain.bigram_rows(s, buckets, mp, mc))] for s in seqs]
    slots, at = [4, 1, 2], [0, 0, 0]
    state = torch.full((5, 1), 77, dtype=torch.int32, device="cuda")
    for q_lens in ([1, 20, 2], [17, 1, 1], [1, 1, 1], [21, 1, 27]):
        ctx = packed(q_lens, slots, at)
        ids = [t for s, a, n in zip(seqs, at, q_lens) for t in s[a:a + n]]
        got = hyper.bigram_embedding(torch.tensor(ids, dtype=torch.int32, device="cuda"), emb.cuda(), 1.5,
                                     table.cuda(), buckets, mp, mc, state, ctx)
        close(got, torch.cat([w[a:a + n] for w, a, n in zip(want, at, q_lens)]), 1e-5)
        at = [a + n for a, n in zip(at, q_lens)]
        assert state[:, 0].tolist() == [77, seqs[1][at[1] - 1], seqs[2][at[2] - 1], 77, seqs[0][at[0] - 1]]


@pytest.mark.parametrize("nq, nk, D, n, neighbours", [
    (3, 3, 12, 4, False), (2, 1, 16, 8, False), (2, 2, 10, 3, True), (1, 1, 128, 64, False),
    (4, 2, 14, 3, False), (2, 2, 20, 0, False)])
def test_rotation_in_place(nq, nk, D, n, neighbours):
    from ginfer_b200.ops import rotary
    g = torch.Generator().manual_seed(D)
    q_off, k_off = 4, 8 + nq * D
    ld = k_off + nk * D + 4
    ld += -ld % 4
    T = 9
    p = torch.randn(T, ld, generator=g)
    freqs = torch.rand(n, generator=g).float() if n else None
    ctx = packed([4, 5], [0, 1], [700, 0])
    want = p.double().clone()
    for off, heads, f in ((q_off, nq, 1.0), (k_off, nk, 0.25)):
        x = want[:, off:off + heads * D].reshape(T, heads, D)
        y = x.clone()
        a = ctx.positions.cpu().double()[:, None] * (freqs.double() if n else torch.zeros(0, dtype=F64))
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        one = slice(0, 2 * n, 2) if neighbours else slice(0, n)
        two = slice(1, 2 * n, 2) if neighbours else slice(n, 2 * n)
        y[..., one], y[..., two] = x[..., one] * c - x[..., two] * s, x[..., two] * c + x[..., one] * s
        want[:, off:off + heads * D] = (y * f).reshape(T, heads * D)
    d = p.cuda()
    rotary.heads_(d, nq, nk, D, q_off, k_off, freqs.cuda() if n else None, neighbours, 0.25, ctx)
    close(d, want, 1e-4)


@pytest.mark.parametrize("act", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh, nkv, hd, vd, kd, kv, n, neighbours", [
    (4, 2, 16, 12, 64, 64, 4, True), (3, 1, 14, 9, 14, 9, 3, True), (2, 2, 32, 32, 32, 32, 16, False),
    (2, 1, 24, 28, 64, 64, 12, True), (1, 1, 8, 8, 16, 16, 0, True), (6, 3, 8, 24, 8, 24, 2, False)])
def test_biases_rotation_and_cache_write(nh, nkv, hd, vd, kd, kv, n, neighbours, act):
    from ginfer_b200.ops import rotary
    g = torch.Generator().manual_seed(hd + vd)
    T, cols = 7, nh * hd + nkv * (hd + vd)
    ld = cols + (-cols % 8) + 8
    p, bias = torch.randn(T, ld, generator=g), torch.randn(cols, generator=g)
    freqs = torch.rand(n, generator=g).float() if n else None
    slots = torch.tensor([5, 0, 30, 2, 9, 11, 3], dtype=torch.int32)
    ctx = packed([7], [0], [333])
    y = p[:, :cols].double() + bias.double()
    q = y[:, :nh * hd].reshape(T, nh, hd)
    k = y[:, nh * hd:(nh + nkv) * hd].reshape(T, nkv, hd)
    v = y[:, (nh + nkv) * hd:].reshape(T, nkv, vd)
    a = ctx.positions.cpu().double()[:, None] * (freqs.double() if n else torch.zeros(0, dtype=F64))
    c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
    one = slice(0, 2 * n, 2) if neighbours else slice(0, n)
    two = slice(1, 2 * n, 2) if neighbours else slice(n, 2 * n)

    def turn(x):
        o = x.clone()
        o[..., one], o[..., two] = x[..., one] * c - x[..., two] * s, x[..., two] * c + x[..., one] * s
        return o

    def wide(x, size):
        return torch.cat([x, torch.zeros(*x.shape[:2], size - x.shape[2], dtype=F64)], -1)
    kp = torch.full((4, 8, nkv, kd), 7.0, dtype=act, device="cuda")
    vp = torch.full((4, 8, nkv, kv), 7.0, dtype=act, device="cuda")
    tol = 1e-4 if act == torch.float32 else 2e-2
    got = rotary.write(p.cuda(), nh, nkv, hd, vd, kd, kv, (0, nh * hd, (nh + nkv) * hd), bias.cuda(),
                       freqs.cuda() if n else None, neighbours, ctx.positions, slots.cuda(), kp, vp, act)
    close(got.view(T, nh, kd), wide(turn(q), kd), tol)
    close(kp.view(32, nkv, kd)[slots.long()], wide(turn(k), kd), tol)
    close(vp.view(32, nkv, kv)[slots.long()], wide(v, kv), tol)
    rest = [i for i in range(32) if i not in slots.tolist()]
    assert float((kp.view(32, -1)[rest] - 7.0).abs().max()) == 0.0
    bare = rotary.write(p.cuda(), nh, nkv, hd, vd, kd, kv, (0, nh * hd, (nh + nkv) * hd), None,
                        freqs.cuda() if n else None, neighbours, ctx.positions, None, kp, vp, act)
    close(bare.view(T, nh, kd), wide(turn(q - bias[:nh * hd].double().view(nh, hd)), kd), tol)


@pytest.mark.parametrize("E, identity, top, groups, keep", [
    (7, 2, 2, 3, 2), (4, 4, 3, 4, 2), (5, 0, 1, 1, 1), (16, 4, 3, 2, 1), (250, 6, 8, 16, 3), (33, 3, 20, 4, 3),
    (1, 1, 2, 1, 1), (3, 5, 4, 2, 1)])
def test_routing_in_groups(E, identity, top, groups, keep):
    from ginfer_b200.ops import moe
    g = torch.Generator().manual_seed(E)
    T, n = 37, E + identity
    z = torch.randn(T, n + 3, generator=g) * 2.0
    corr = torch.randn(n, generator=g) * 0.3 - 0.4       # most choice scores are negative
    idx, wgt, idw, gate = moe.route_grouped(z.cuda(), E, identity, top, corr.cuda(), groups, keep, n + 1)
    s = torch.softmax(z[:, :n].double(), -1)
    for t in range(T):
        want = plain.choose(s[t], corr.double(), top, {"count": groups, "keep": keep})
        assert idx[t].tolist() == [e if e < E else -1 for e in want], t
        close(wgt[t], torch.stack([s[t, e] if e < E else torch.zeros((), dtype=F64) for e in want]), 1e-6)
        if identity:
            close(idw[t], sum([s[t, e] for e in want if e >= E], torch.zeros((), dtype=F64)), 1e-6)
    assert identity or idw is None
    close(gate, torch.sigmoid(z[:, n + 1].double()), 1e-6)
    more, w2, _, none = moe.route_grouped(z.cuda(), E, identity, top, corr.cuda(), groups, keep, n + 1, 3)
    assert none is None and torch.equal(more[:, :top], idx) and torch.equal(w2[:, :top], wgt)
    assert more[:, top:].tolist() == [[E, E + 1, E + 2]] * T
    assert torch.equal(w2[:, top:], gate[:, None].expand(-1, 3))
    with pytest.raises(ValueError):
        moe.route_grouped(z.cuda(), E, identity, n + 1, corr.cuda(), groups, keep)


def test_ties_go_to_the_lower_index():
    from ginfer_b200.ops import moe
    idx, _, idw, _ = moe.route_grouped(torch.zeros(5, 12, device="cuda"), 10, 2, 4, None, 3, 2)
    assert idx.tolist() == [[0, 1, 2, 3]] * 5 and float(idw.abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("SF", [80, 96, 48])
@pytest.mark.parametrize("T", [1, 3, 40, 700])
def test_routed_feed_forward_with_identities_and_a_shared_expert(T, SF, dtype):
    """The whole part, its sum formed by itself (``materialize``), on every kind of grouped product (a
    handful of pairs, tiles, the persistent kernel); also when every token chooses identities only; a
    shared expert with products of its own and one that is as large as one or two experts."""
    from ginfer_b200.parts import PartSpec, make_part
    g = torch.Generator().manual_seed(T)
    W, F, E, I = 64, 48, 6, 2
    part = make_part("feed_forward", PartSpec("group_routed_glu", dict(
        hidden_size=W, intermediate_size=F, num_experts=E, top_k=2, identity=I, groups=4, keep_groups=2,
        shared_size=SF)))
    t = {s.name: torch.randn(s.shape, generator=g) * (s.shape[-1] ** -0.5 if len(s.shape) == 2 else 0.2)
         for s in part.tensor_specs()}
    assert part.always == (SF // F if SF % F == 0 else 0)
    t["mlp.router"] *= 6.0
    x = torch.randn(T, W, generator=g)
    for only_identity in (False, True):
        if only_identity:
            t["mlp.correction"] = torch.tensor([0.0] * E + [9.0] * I)
        kept = {k: v.to(dtype) if v.dim() == 2 else v for k, v in t.items()}
        part.load({k: v.cuda() for k, v in kept.items()}, dtype, torch.device("cuda"))
        got = part.forward(x.to(dtype).cuda(), None)
        m = {"router": {"experts": E, "top": 2, "groups": {"count": 4, "keep": 2}}, "shared": {"ff": SF}}
        want = plain.routed(x.to(dtype).double(), {k: v.double() for k, v in kept.items()}, "mlp.", m,
                            bf16 if dtype == torch.bfloat16 else plain.same)
        err = (got.double().cpu() - want).norm(dim=1) / want.norm(dim=1)
        assert float(err.median()) <= (1e-5 if dtype == torch.float32 else 0.02)
        assert int((err > (1e-4 if dtype == torch.float32 else 0.05)).sum()) <= T // 50


@pytest.mark.parametrize("H, D, Vd", [(3, 8, 12), (2, 10, 9), (2, 128, 64), (1, 36, 200), (4, 7, 5),
                                      (2, 64, 32), (1, 256, 16), (4, 16, 128), (2, 128, 128)])
def test_memory_gates_recurrence_and_normaliser(H, D, Vd):
    """Gates, states and read-outs of the matrix memory for two requests under cuts of every kind, and the
    gated norm behind them."""
    from ginfer_b200.ops import decay
    g = torch.Generator().manual_seed(D + Vd)
    lens, slots, cap = [190, 61], [2, 0], 4.0
    HD, HV = H * D, H * Vd
    cols = 2 * HD + 2 * HV + 2 * H
    ld = cols + (-cols % 8)
    ib, fb = torch.randn(H, generator=g), torch.randn(H, generator=g) + 2.0
    norm = 1.0 + 0.2 * torch.randn(HV, generator=g)
    cases = [torch.randn(n, ld, generator=g) for n in lens]
    for c in cases:
        c[:, 2 * HD + 2 * HV:] *= 3.0
    wants = []
    for c in cases:
        p, T = c.double(), c.shape[0]
        i = plain.capped(p[:, cols - 2 * H:cols - H] + ib.double(), cap)
        f = plain.log_sigmoid(plain.capped(p[:, cols - H:cols] + fb.double(), cap))
        q = p[:, :HD].reshape(T, H, D) * D ** -0.5
        k, v = p[:, HD:2 * HD].reshape(T, H, D), p[:, 2 * HD:2 * HD + HV].reshape(T, H, Vd)
        o = torch.stack([plain.matrix_memory_head(q[:, n], k[:, n], v[:, n], i[:, n], f[:, n])
                         for n in range(H)], 1)
        y = plain.rms_norm(o, 1e-5).reshape(T, HV) * norm.double() * torch.sigmoid(
            p[:, 2 * HD + HV:2 * HD + 2 * HV])
        wants.append(y)
    n_off = HD * Vd
    for steps in ([[190, 61]], [[70, 1], [1, 1], [1, 40], [2, 2], [103, 17], [13, 0]],
                  [[1, 1]] * 6 + [[2, 3], [182, 52]]):
        state = torch.zeros(4, n_off + HD + H, device="cuda")
        state[1] = state[3] = 5.0
        at = [0, 0]
        for q_lens in steps:
            ids = [b for b in range(2) if q_lens[b]]
            ctx = packed([q_lens[b] for b in ids], [slots[b] for b in ids])
            rows = [slice(at[b], at[b] + q_lens[b]) for b in ids]
            p = torch.cat([cases[b][r] for b, r in zip(ids, rows)]).cuda()
            keep, write, m = decay.memory_gates(p, cols - 2 * H, cols - H, ib.cuda(), fb.cuda(), cap, state,
                                                n_off + HD, ctx, H)
            assert float(keep.max()) <= 1.0 + 1e-5 and float(write.max()) <= 1.0 + 1e-5
            o, nq = decay.recurrence(p[:, :HD], p[:, HD:2 * HD], p[:, 2 * HD:2 * HD + HV], keep, state, ctx,
                                     H, H, D, Vd, k_scale=write, normaliser=n_off)
            y = decay.gated_norm(o, p[:, 2 * HD + HV:2 * HD + 2 * HV], norm.cuda(), Vd, False, 1e-5,
                                 torch.float32, sigmoid_gate=True, normaliser=(nq, m, D ** -0.5, 1e-6))
            close(y, torch.cat([wants[b][r] for b, r in zip(ids, rows)]), 3e-3)
            at = [a + n for a, n in zip(at, q_lens)]
        assert at == lens
        assert float((state[[1, 3]] - 5.0).abs().max()) == 0.0


@pytest.mark.parametrize("hd, nh, nkv, page", [(16, 4, 2, 16), (48, 6, 2, 8), (64, 4, 1, 16), (64, 8, 8, 16),
                                               (80, 2, 2, 16), (128, 4, 2, 32), (128, 16, 2, 16)])
def test_attention_with_a_sink_a_head(hd, nh, nkv, page):
    """Prompts, later portions, single tokens and both together over shuffled pages, every merge of the
    split decode kernels; sinks from nothing to far above every score."""
    from ginfer_b200 import ops
    from ginfer_b200.ops import attention_bf16
    g = torch.Generator().manual_seed(hd * nh)
    kv_lens, q_lens = [300, 150, 77, 1], [300, 1, 40, 1]
    n_pages = sum(-(-n // page) for n in kv_lens)
    perm = torch.randperm(n_pages, generator=g)
    width = max(-(-n // page) for n in kv_lens)
    table = torch.full((4, width), -1, dtype=torch.int32)
    at = 0
    for b, n in enumerate(kv_lens):
        c = -(-n // page)
        table[b, :c] = perm[at:at + c].to(torch.int32)
        at += c
    pages = torch.randn(2, n_pages, page, nkv, hd, generator=g).to(torch.bfloat16)
    sinks = torch.linspace(-30.0, 12.0, nh)
    scale = 2.0 * hd ** -0.5

    def run(ids, lens):
        ctx = packed(lens, ids, [kv_lens[b] - n for b, n in zip(ids, lens)])
        ctx.kv_lens = torch.tensor([kv_lens[b] for b in ids], dtype=torch.int32, device="cuda")
        ctx.max_kv_len = max(kv_lens[b] for b in ids)
        q = torch.randn(sum(lens), nh * hd, generator=g).to(torch.bfloat16)
        want = torch.zeros(sum(lens), nh, hd, dtype=F64)
        r = 0
        for b, n in zip(ids, lens):
            flat = table[b, :-(-kv_lens[b] // page)].long()
            K, V = (pages[i][flat].reshape(-1, nkv, hd)[:kv_lens[b]].double() for i in (0, 1))
            for i in range(n):
                p = kv_lens[b] - n + i
                for h in range(nh):
                    s = (K[:p + 1, h // (nh // nkv)] @ q[r, h * hd:(h + 1) * hd].double()) * scale
                    want[r, h] = plain.softmax_with_sink(s[None], sinks[h].double())[0] @ \
                        V[:p + 1, h // (nh // nkv)]
                r += 1
        args = (q.cuda(), pages.cuda(), table[torch.tensor(ids)].cuda(), ctx, nh, nkv, hd, scale, 0, page)
        return args, want.reshape(-1, nh * hd)
    for ids, lens in (([0, 2], [300, 40]), ([1, 0], [1, 130]), ([1, 3, 0], [1, 1, 1])):
        args, want = run(ids, lens)
        close(ops.paged_attention(*args, sink=sinks.cuda()), want, 2e-2)
        f = ops.paged_attention_simt(*args[:3], args[3].seq_of_token, args[3].positions, nh, nkv, hd, scale, 0,
                                     page, sink=sinks.cuda())
        close(f, want, 2e-2)
        if max(lens) == 1:
            for splits in (1, 2, 4, 8, 3):
                for scratch in (False, True):
                    y = attention_bf16.decode(args[0], args[1], args[2], args[3].cu_seqlens_q,
                                              args[3].positions, len(ids), nh, nkv, hd, scale, 0, page, splits,
                                              through_scratch=scratch, sink=sinks.cuda(), use_tma=not scratch)
                    close(y, want, 2e-2)
            if attention_bf16.tma_serves(hd, page, 8):
                y = attention_bf16.decode(args[0], args[1], args[2], args[3].cu_seqlens_q, args[3].positions,
                                          len(ids), nh, nkv, hd, scale, 0, page, 8, parts=2, sink=sinks.cuda())
                close(y, want, 2e-2)


@pytest.mark.parametrize("H, G, D, Vd", [(3, 3, 32, 64), (4, 2, 20, 36), (2, 1, 128, 132), (2, 2, 64, 200),
                                         (1, 1, 100, 8), (6, 3, 4, 4)])
def test_a_chunk_of_tokens_at_a_time(monkeypatch, H, G, D, Vd):
    """Long portions in chunks against token by token and against the equations, in one batch with short
    portions and single tokens in front and behind, from states that are not zero; keys shared by groups of
    heads, step factors, a skip, a normaliser; decays of zero, of one and of 1e-30."""
    from ginfer_b200.ops import decay
    g = torch.Generator().manual_seed(D * Vd)
    lens, slots = [1, 1, 130, 5, 64, 1, 257], [6, 0, 3, 1, 7, 2, 4]
    T = sum(lens)
    n_off = H * D * Vd
    q, k = torch.randn(T, G * D, generator=g), torch.randn(T, G * D, generator=g) * D ** -0.5
    v, c = torch.randn(T, H * Vd, generator=g), torch.rand(T, H, generator=g)
    decays = 1.0 - torch.rand(T, H, generator=g) ** 4
    decays[::17], decays[5::31], decays[3::29] = 1.0, 0.0, 1e-30
    skip = torch.randn(H, generator=g)
    start = torch.randn(8, n_off + H * D + 3, generator=g)
    ctx = packed(lens, slots)
    got = {}
    for name, limit in (("chunks", 64), ("tokens", 1 << 30)):
        monkeypatch.setattr(decay, "CHUNK_MIN_TOKENS", limit)
        a, b = start.cuda(), start.cuda()
        args = [t.cuda() for t in (q, k, v, decays)]
        plain_o = decay.recurrence(*args, a, ctx, H, G, D, Vd, k_scale=c.cuda(), skip=skip.cuda())
        o, nq = decay.recurrence(*args, b, ctx, H, G, D, Vd, normaliser=n_off)
        got[name] = [t.double().cpu() for t in (plain_o, a, o, nq, b)]
    for x, y in zip(got["chunks"], got["tokens"]):
        assert float((x - y).abs().max()) <= 2e-5 * float(y.abs().max())
    # against the equations: the request of 130 tokens
    at, n, s = sum(lens[:2]), lens[2], slots[2]
    for h in range(H):
        S = start[s, h * D * Vd:(h + 1) * D * Vd].double().view(D, Vd)
        z = start[s, n_off + h * D:n_off + (h + 1) * D].double()
        for t in range(at, at + n):
            kk = k[t, (h // (H // G)) * D:][:D].double()
            qq = q[t, (h // (H // G)) * D:][:D].double()
            S = decays[t, h].double() * S + torch.outer(kk, v[t, h * Vd:(h + 1) * Vd].double())
            z = decays[t, h].double() * z + kk
            close(got["chunks"][2][t, h * Vd:(h + 1) * Vd], S.T @ qq, 2e-4)
            close(got["chunks"][3][t, h], z @ qq, 2e-4)
        close(got["chunks"][4][s, h * D * Vd:(h + 1) * D * Vd].view(D, Vd), S, 2e-4)
        close(got["chunks"][4][s, n_off + h * D:n_off + (h + 1) * D], z, 2e-4)
    # slots that no request of the step has, and what lies behind the states, stay as they were
    assert torch.equal(got["chunks"][4][5], start[5].double())
    assert torch.equal(got["chunks"][4][:, n_off + H * D:], start[:, n_off + H * D:].double())
