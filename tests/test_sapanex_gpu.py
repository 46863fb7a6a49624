"""The Sapanex decoder through the engine, and each of its mechanisms alone (GPU), against the plain 64-bit statement in
plain_sapanex.py.  The configurations are in sapanex_cases.py: K (odd sizes, exact kernels), L (the tensor-core kernels'
sizes), M (everything plural is one), N (recurrences only), O (attention only: no window, no rotation), P (groups of 32 and
20 heads, pages of 32, blocks that do not divide a page).
"""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_sapanex as plain
import sapanex_cases as cases
from helpers import ROOT, Trace, assert_close, check_trace, random_tokens, run_trace_inprocess

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
NAMES = ("K", "L", "M", "N", "O", "P")
ENGINE_CASES = [(n, d) for n in NAMES for d in ("float32", "bfloat16")]


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return str(tmp_path_factory.mktemp("sapanex"))


def stored(dtype):
    return torch.bfloat16 if dtype == "bfloat16" else torch.float32


def runner_for(root, name, dtype, pages=64, requests=4, page=None):
    from inferloop_b200.engine import ModelRunner
    return ModelRunner.from_folder(cases.folder(root, name, stored(dtype)), dtype=dtype, device=DEV, page_size=page or cases.CASES[name][2],
                                   num_pages=pages, max_requests=requests)


def tokens_for(name, n, seed):
    return random_tokens(n, cases.CASES[name][0]["vocab"], seed)


def reference(root, name, dtype, tokens):
    return cases.plain_model(root, name, stored(dtype)).forward(tokens)


# a position's logits pass several layers that amplify what bfloat16 rounds (norms of sums, a softmax that picks single keys)
BF16 = 3e-2
F32_OF_MAX = 3e-5


def close(got, ref, dtype, what):
    if dtype == "float32":
        got, ref = got.double().cpu(), ref.double().cpu()
        err = (got - ref).abs().max()
        assert torch.isfinite(got).all() and err <= F32_OF_MAX * ref.abs().max(), f"{what}: {float(err):.3e} of {float(ref.abs().max()):.3e}"
    else:
        assert_close(got, ref, dtype, what, bf16_rel_of_max=BF16)


def check(out, t, ref, dtype, what):
    for step, rows in t.rows.items():
        close(torch.from_numpy(out[step]), torch.stack([ref[rid][pos] for rid, pos in rows]), dtype, f"{what} step {step} rows {rows[:4]}...")


# ------------------------------------------------------------------------------ the engine
@pytest.mark.parametrize("name,dtype", ENGINE_CASES)
def test_whole_prompt_and_every_layer(root, name, dtype):
    """One prompt in one step: the residual stream after every layer, and all logits."""
    from inferloop_b200.engine import StepEntry
    r = runner_for(root, name, dtype)
    toks = tokens_for(name, 120, 1)
    per_layer = []
    ref = cases.plain_model(root, name, stored(dtype)).forward(toks, per_layer)
    got = []
    for b in r.model.blocks:
        def hooked(hidden, step, cache, orig=b.forward):
            orig(hidden, step, cache)
            got.append(hidden.cpu().clone())
        b.forward = hooked
    logits = r.step([StepEntry("a", toks, list(range(len(toks))))])
    assert len(got) == len(per_layer) == len(cases.CASES[name][0]["layers"])
    for i, (g, w) in enumerate(zip(got, per_layer)):
        close(g, w, dtype, f"{name} layer {i}")
    close(logits, ref, dtype, f"{name} logits")


@pytest.mark.parametrize("name,dtype", ENGINE_CASES)
def test_prefill_against_token_by_token_and_portions(root, name, dtype):
    """The same sequence token by token from the first token on, and in portions of changing size down to two tokens with the
    last tokens one by one."""
    toks = tokens_for(name, 130, 2)
    ref = {"a": reference(root, name, dtype, toks)}
    r = runner_for(root, name, dtype, pages=80)
    t = Trace()
    for i, tok in enumerate(toks):
        t.step([("a", [tok], [0])], end=["a"] if i == len(toks) - 1 else [])
    check(run_trace_inprocess(r, t), t, ref, dtype, f"{name} token by token")
    t = Trace()
    at = 0
    for n in (2, 5, 3, 17, 2, 9, 16, 1, 2, 33, 7, 2):
        t.step([("a", toks[at:at + n], list(range(n)))])
        at += n
    while at < len(toks):
        t.step([("a", toks[at:at + 1], [0])], end=["a"] if at == len(toks) - 1 else [])
        at += 1
    check(run_trace_inprocess(r, t), t, ref, dtype, f"{name} portions")
    r.cache.check()
    assert all(n == g.pool.num_pages for g, n in zip(r.cache.groups, r.cache.free_pages().values()))


@pytest.mark.parametrize("name,dtype", ENGINE_CASES)
def test_mixed_batches_with_pages_and_slots_used_again(root, name, dtype):
    """Up to four live requests of unequal length, portions beside single tokens, four state slots for seven requests and a
    pool that cannot hold all of them: what ends gives its pages (of both kinds) and its slot to the next.  Every row
    equals the request alone."""
    lens = {"a": 97, "b": 5, "c": 124, "d": 21, "e": 110, "f": 2, "g": 83}
    toks = {k: tokens_for(name, n, 50 + i) for i, (k, n) in enumerate(lens.items())}
    ref = {k: reference(root, name, dtype, v) for k, v in toks.items()}
    page = cases.CASES[name][2]
    pages = sum(-(-n // page) for n in (97, 124, 110, 21)) + 1
    r = runner_for(root, name, dtype, pages=pages, requests=4)
    t = Trace()
    cursor = {k: 0 for k in lens}
    waiting, live = list(lens), []
    portion = {"a": [2, 66, 3], "b": [5], "c": [31, 2, 70], "d": [8, 8], "e": [3, 90], "f": [2], "g": [60]}
    step = 0
    while waiting or live:
        while waiting and len(live) < 4:
            if sum(-(-lens[k] // page) for k in live + [waiting[0]]) > pages:
                break
            live.append(waiting.pop(0))
        entries, ended = [], []
        for k in live:
            n = min(portion[k].pop(0) if portion[k] else 1, lens[k] - cursor[k])
            entries.append((k, toks[k][cursor[k]:cursor[k] + n], sorted({0, n // 2, n - 1})))
            cursor[k] += n
            if cursor[k] == lens[k]:
                ended.append(k)
        t.step(entries, end=ended)
        live = [k for k in live if k not in ended]
        step += 1
        assert step < 500
    check(run_trace_inprocess(r, t), t, ref, dtype, f"{name} mixed")
    info = r.cache.inspect()
    assert info["begun"] == len(lens) and info["live_requests"] == 0
    for g in info["groups"]:
        assert g["reuses"] > 0, "no page was used again"
    r.cache.check()


@pytest.mark.parametrize("name,dtype", [("K", "float32"), ("L", "bfloat16"), ("M", "float32"), ("P", "bfloat16"), ("O", "bfloat16")])
def test_long_decoding_through_recorded_graphs(root, name, dtype):
    """A short prompt, then hundreds of single tokens (recorded decode graphs after the first): blocks are completed, become
    visible and outlive their tokens' pages while decoding."""
    toks = tokens_for(name, 420, 3)
    ref = {"a": reference(root, name, dtype, toks)}
    r = runner_for(root, name, dtype, pages=-(-430 // cases.CASES[name][2]))
    t = Trace()
    t.step([("a", toks[:20], [19])])
    for i in range(20, len(toks)):
        t.step([("a", [toks[i]], [0])], end=["a"] if i == len(toks) - 1 else [])
    check(run_trace_inprocess(r, t), t, ref, dtype, f"{name} long decoding")
    assert r.graphs is not None and r.graphs.whole and r.graphs.replays > 350
    if any(g.need.window is not None for g in r.cache.groups):
        assert r.cache.stats["window_pages_released"] > 0


@pytest.mark.parametrize("name,dtype", [("K", "float32"), ("L", "float32"), ("L", "bfloat16"), ("N", "bfloat16"), ("P", "bfloat16"), ("M", "float32")])
def test_a_long_prompt_whole_and_in_portions(root, name, dtype):
    """700 tokens in one step (recurrences in chunks, pooled rows over several key tiles) against the plain statement, and in
    portions of 128, 100 and 37: the logits at a position do not depend on the cut."""
    from inferloop_b200.engine import StepEntry
    toks = tokens_for(name, 700, 77)
    want = list(range(5, 700, 10)) + [699]
    r = runner_for(root, name, dtype, pages=-(-700 // cases.CASES[name][2]) + 2)
    whole = r.step([StepEntry("w", toks, want)]).float().cpu().clone()
    r.end("w")
    close(whole, reference(root, name, dtype, toks)[want], dtype, f"{name} 700 tokens whole")
    for portion in (128, 100, 37):
        rows = []
        for at in range(0, 700, portion):
            part = toks[at:at + portion]
            rows.append(r.step([StepEntry("p", part, [w - at for w in want if at <= w < at + len(part)])]).float().cpu().clone())
        r.end("p")
        close(torch.cat(rows), whole, dtype, f"{name} portions of {portion} against the whole prompt")


@pytest.mark.parametrize("name,dtype", [("K", "float32"), ("L", "bfloat16"), ("M", "float32"), ("O", "float32")])
def test_greedy_generation_through_the_entry_point(root, name, dtype):
    from inferloop_b200 import Engine, SamplingParams
    page = cases.CASES[name][2]
    model = cases.plain_model(root, name, stored(dtype))
    prompts = [tokens_for(name, n, 30 + n) for n in (3, 12, 31, 64)]
    engine = Engine(cases.folder(root, name, stored(dtype)), dtype=dtype, block_size=page, num_gpu_blocks_override=96,
                    max_num_seqs=4, prefill_chunk_tokens=32, max_num_batched_tokens=40)
    got = engine.generate(prompts, SamplingParams(), max_new_tokens=12)
    for p, g in zip(prompts, got):
        assert len(g) == 12
        ref = model.forward(list(p) + list(g))[len(p) - 1:-1]
        bound = (BF16 if dtype == "bfloat16" else F32_OF_MAX) * float(ref.abs().max())
        for i, tok in enumerate(g):        # teacher-forced: every chosen token is the best one within the bound
            assert ref[i, tok] >= ref[i].max() - 2 * bound
    info = engine.inspect()
    assert info["running"] == 0 and all(g["free"] == g["total"] for g in info["cache"]["groups"])


def test_pools_sized_from_memory_and_generation_from_a_mapping():
    """The engine with pools of its own choosing (a pooled group gets a page per page_size * pool tokens) and random weights."""
    from inferloop_b200 import Engine, SamplingParams
    engine = Engine(cases.CONFIG_L, random_weights_seed=3, dtype="bfloat16", block_size=16, max_num_seqs=3, max_model_len=512,
                    prefill_chunk_tokens=64, gpu_memory_utilization=0.2)
    groups = engine.runner.cache.groups
    tokens = {(g.need.kv_heads, g.need.head_dim): g.pool.num_pages for g in groups if g.need.stride == 1}
    for g in groups:
        if g.need.stride > 1:
            assert g.pool.num_pages >= 3 * (512 // g.need.stride // 16) and g.pool.num_pages < 512 * 3
    assert len(tokens) == 3
    assert [len(x) for x in engine.generate([[1, 2, 3], list(range(40))], SamplingParams(), max_new_tokens=5)] == [5, 5]


def test_the_command_line_generates_from_a_sapanex_folder(root):
    name, dtype = "M", "float32"
    prompt = tokens_for(name, 9, 41)
    out = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "infer"), "generate", cases.folder(root, name, stored(dtype)),
                          "--tokens", ",".join(map(str, prompt)), "--max-new-tokens", "6", "--dtype", dtype, "--block-size", "16",
                          "--num-gpu-blocks-override", "8"], capture_output=True, text=True, timeout=900)
    assert out.returncode == 0, out.stderr
    got = json.loads(out.stdout.strip().splitlines()[-1])["tokens"]
    ref = reference(root, name, dtype, list(prompt) + got)[len(prompt) - 1:-1]
    for i, tok in enumerate(got):
        assert ref[i, tok] >= ref[i].max() - 2 * F32_OF_MAX * float(ref.abs().max())


def test_the_trace_program_replays_a_sapanex_folder(root, tmp_path):
    name, dtype = "K", "float32"
    toks = {"x": tokens_for(name, 40, 5), "y": tokens_for(name, 9, 6)}
    ref = {k: reference(root, name, dtype, v) for k, v in toks.items()}
    t = Trace()
    t.step([("x", toks["x"][:33], [0, 32]), ("y", toks["y"][:2], [1])])
    t.step([("x", toks["x"][33:34], [0]), ("y", toks["y"][2:], [0, 6])], end=["y"])
    for i in range(34, 40):
        t.step([("x", toks["x"][i:i + 1], [0])], end=["x"] if i == 39 else [])
    cmd = [sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", cases.folder(root, name, stored(dtype)), "--dtype", dtype,
           "--out", str(tmp_path), "--max-tokens", "128", "--block-size", "4"]
    proc = subprocess.run(cmd, input=t.lines(), capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr
    vocab = cases.CASES[name][0]["vocab"]
    out = {s: np.fromfile(os.path.join(str(tmp_path), f"{s}.f32"), dtype="<f4").reshape(len(rows), vocab) for s, rows in t.rows.items()}
    check(out, t, ref, dtype, "trace program")


# ------------------------------------------------------------------------------ each mechanism alone
class FakeStep:
    """The device arrays of a batch, for kernels called without an engine: sequences of `lens` tokens that start at `starts`,
    in slots `slots`."""

    def __init__(self, lens, starts, slots=None):
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
        self.h_q_len = list(lens)
        self.n_seqs, self.n_tokens = len(lens), sum(lens)
        self.max_q_len = max(lens)
        self.decode_only = all(n == 1 for n in lens)
        self.cu_q = i32([sum(lens[:i]) for i in range(len(lens) + 1)])
        self.positions = i32([s + j for n, s in zip(lens, starts) for j in range(n)])
        self.seq_of_token = i32([i for i, n in enumerate(lens) for _ in range(n)])
        self.slots = i32(slots if slots is not None else list(range(len(lens))))
        self.h_kv_len = [s + n for n, s in zip(lens, starts)]
        self.max_kv_len = max(self.h_kv_len)
        self.position_tables = {}


def f32(t):
    return t.float().to(DEV).contiguous()


@pytest.mark.parametrize("width", [1, 50, 256, 4100, 6000])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_norm_of_a_sum(width, dtype):
    """Rows on 16-byte boundaries and others, rows longer than the registers keep; the stream, its copy and what the next
    sublayer adds into from one read; without the stream."""
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    T, alpha = 9, 1.75
    x, w = 2 * torch.randn(T, width, generator=g), 1 + 0.2 * torch.randn(width, generator=g)
    hidden, xc, y = f32(x), torch.empty(T, width, dtype=dtype, device=DEV), torch.empty(T, width, device=DEV)
    ops.cast_zero(hidden, xc, y, alpha)
    assert torch.equal(y.cpu(), (x * alpha)) and torch.equal(xc.cpu(), x.to(dtype))
    ops.cast_zero(hidden, xc, y)
    assert float(y.abs().max()) == 0.0
    s = torch.randn(T, width, generator=g) * 3
    ref = plain.rms(s.double(), 1e-3) * w.double()
    for keep_stream in (True, False):
        y.copy_(s.to(DEV))
        hidden.fill_(7.0)
        ops.sum_norm(y, f32(w), 1e-3, alpha, hidden if keep_stream else None, xc)
        assert_close(xc, ref, "float32" if dtype == torch.float32 else "bfloat16", "copy")
        assert_close(y, alpha * ref, "float32", "next sum")
        if keep_stream:
            assert_close(hidden, ref, "float32", "stream")
        else:
            assert float(hidden.min()) == 7.0


@pytest.mark.parametrize("rows,width,pad", [(5, 7, 3), (33, 64, 0), (300, 128, 8), (1, 1000, 24)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_tanh_and_relu_squared_of_rows(rows, width, pad, dtype):
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    x = (2 * torch.randn(rows, width + pad, generator=g)).to(dtype)
    for act, f in (("tanh", torch.tanh), ("relu2", lambda v: torch.relu(v) ** 2)):
        out = torch.empty(rows, width, dtype=dtype, device=DEV)
        xd = x.to(DEV)
        ops.act_rows(xd[:, :width], act, out)
        ref = f(x.double()[:, :width])
        assert (out.double().cpu() - ref).abs().max() <= (2e-6 if dtype == torch.float32 else 2.0 ** -8) * max(1.0, float(ref.abs().max()))
        ops.act_rows(xd[:, :width], act, xd[:, :width])
        assert torch.equal(xd[:, :width], out) and torch.equal(xd[:, width:].cpu(), x[:, width:])


@pytest.mark.parametrize("M", [1, 3, 8, 17, 64, 100, 128, 200, 513, 2048])
@pytest.mark.parametrize("N,K", [(384, 256), (1000, 72), (4096, 1024)])
def test_relu_squared_in_the_products_epilogue(M, N, K):
    """Every form of the tensor-core product (few tokens, clusters, many tokens, pairs of CTAs) squares once, before the one
    rounding; a product without it is as it was."""
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(M + N)
    a = torch.randn(M, K, generator=g).to(torch.bfloat16)
    w = (torch.randn(N, K, generator=g) / math.sqrt(K)).to(torch.bfloat16)
    ref = a.double() @ w.double().T
    for pairs in (0, 1, 2):
        ops.gemm_pairs(pairs)
        try:
            out = torch.full((M, N), 9.0, dtype=torch.bfloat16, device=DEV)
            ops.gemm_tc(a.to(DEV), w.to(DEV), out, relu2=True)
            want = torch.relu(ref) ** 2
            assert ((out.double().cpu() - want).abs() <= 2.0 ** -8 * want + 1e-4).all()
            ops.gemm_tc(a.to(DEV), w.to(DEV), out)
            assert ((out.double().cpu() - ref).abs() <= 2.0 ** -8 * ref.abs() + 1e-4).all()
        finally:
            ops.gemm_pairs(1)
    with pytest.raises(ops.KernelError):
        ops.gemm_tc(a.to(DEV), w.to(DEV), torch.empty(M, N, device=DEV), relu2=True)


@pytest.mark.parametrize("heads,dv,pad", [(1, 9, 3), (3, 10, 0), (8, 64, 8), (2, 128, 4), (5, 300, 4)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_norm_of_each_head_with_a_sigmoid_gate(heads, dv, pad, dtype):
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(heads * dv)
    T, width = 11, heads * dv
    y = 3 * torch.randn(T, width, generator=g) * torch.logspace(-2, 2, heads).repeat_interleave(dv)
    z = (2 * torch.randn(T, 8 + width + pad, generator=g)).to(dtype)
    w = 1 + 0.2 * torch.randn(width, generator=g)
    out = torch.empty(T, width, dtype=dtype, device=DEV)
    ops.rms_gate(f32(y), z.to(DEV)[:, 8:], f32(w), 1e-5, out, groups=heads)
    ref = plain.rms(y.double().view(T, heads, dv), 1e-5).reshape(T, width) * w.double() * torch.sigmoid(z.double()[:, 8:8 + width])
    if dtype == torch.float32:
        assert_close(out, ref, "float32", "norm and gate")
    else:
        assert (out.double().cpu() - ref).abs().max() <= 2.0 ** -8 * ref.abs().max()


def test_the_rotations_table_is_stretched():
    from inferloop_b200.config.spec import PartSpec
    from inferloop_b200.parts import registry
    from inferloop_b200.parts.base import BuildContext, Workspace
    ctx = BuildContext(dtype=torch.float32, device=torch.device(DEV), workspace=Workspace(torch.device(DEV)))
    ramp = (8.0, 256.0, 16.0, 1.0)
    a = registry.build("position", PartSpec.make("rope_neox", theta=10000.0, rotary_dim=64, ramp=ramp), ctx)
    b = registry.build("position", PartSpec.make("rope_neox", theta=10000.0, rotary_dim=64), ctx)
    step = FakeStep([5], [1000])
    ta, tb = a.table(step).cpu().double(), b.table(step).cpu().double()          # (two tables of one step live side by side)
    for table, (freq, stretch) in ((ta, plain.frequencies(10000.0, 64, dict(zip(("factor", "original", "fast", "slow"), ramp)))),
                                   (tb, plain.frequencies(10000.0, 64))):
        ang = torch.arange(1000, 1005).double()[:, None] * freq[None, :]
        assert (table[..., 0] - stretch * torch.cos(ang)).abs().max() < 3e-7 and (table[..., 1] - stretch * torch.sin(ang)).abs().max() < 3e-7


def scattered_tables(lens, page, pages, seed, first_free=0):
    """Block tables whose pages lie anywhere in the pool: [seqs, max_blocks] int32, -1 where nothing is held."""
    g = torch.Generator().manual_seed(seed)
    order = torch.randperm(pages, generator=g).tolist()
    width = max(max(-(-n // page) for n in lens), 1) + 3
    table = torch.full((len(lens), width), -1, dtype=torch.int32)
    for i, n in enumerate(lens):
        for b in range(-(-n // page)):
            table[i, b] = order.pop()
    return table


def rows_of(cache, table, page, n):
    """[n, heads, size] rows 0 .. n - 1 of a sequence from the pages, in 64-bit."""
    out = [cache[table[j // page], :, j % page] for j in range(n)]
    return torch.stack(out).double().cpu() if out else torch.zeros(0, cache.shape[1], cache.shape[3], dtype=torch.float64)


@pytest.mark.parametrize("nq,nkv,d,dv,rd,page", [(5, 1, 12, 10, 8, 4), (1, 1, 7, 6, 2, 8), (8, 2, 64, 64, 64, 16), (4, 1, 128, 64, 32, 16), (3, 3, 48, 80, 16, 32)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_norms_over_whole_rows_with_turned_values(nq, nkv, d, dv, rd, page, dtype):
    """q and k normed over all heads at once (heads of very different sizes: a norm a head would show), turned, values turned
    over their whole size, both written to pages anywhere in the pool; no rotation at all; then the heads turned back."""
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(nq * d + dv)
    lens, starts = [37, 1, 9], [5, 60, 0]
    T = sum(lens)
    size = lambda n, w: torch.logspace(-1, 1, n).repeat_interleave(w) if n > 1 else torch.ones(w)
    wide = torch.cat([size(nq, d), size(nkv, d), torch.ones(nkv * dv)])
    qkv = (torch.randn(T, wide.numel() + 5, generator=g) * torch.cat([wide, torch.ones(5)])).to(dtype)
    wq, wk = 1 + 0.3 * torch.randn(nq * d, generator=g), 1 + 0.3 * torch.randn(nkv * d, generator=g)
    freq, stretch = plain.frequencies(50.0, rd, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0})
    vfreq, _ = plain.frequencies(50.0, dv)
    step = FakeStep(lens, starts)
    pos = step.positions.cpu()
    table_of = lambda f, s: f32(torch.stack([torch.cos(pos.double()[:, None] * f) * s, torch.sin(pos.double()[:, None] * f) * s], dim=-1))
    table = scattered_tables([s + n for s, n in zip(starts, lens)], page, 64, 3)
    for turned in (True, False):
        k_cache = torch.full((64, nkv, page, d), 3.0, dtype=dtype, device=DEV)
        v_cache = torch.full((64, nkv, page, dv), 3.0, dtype=dtype, device=DEV)
        q_out = torch.empty(T, nq * d, dtype=dtype, device=DEV)
        ops.rows_norm_rope_cache(qkv.to(DEV), q_out, f32(wq), f32(wk), 1e-4, table_of(freq, stretch) if turned else None, rd,
                                 table_of(vfreq, 1.0) if turned else None, step, table.to(DEV), k_cache, v_cache, nq, nkv, d, dv)
        x = qkv.double()
        q = (plain.rms(x[:, :nq * d], 1e-4) * wq.double()).view(T, nq, d)
        k = (plain.rms(x[:, nq * d:(nq + nkv) * d], 1e-4) * wk.double()).view(T, nkv, d)
        v = x[:, (nq + nkv) * d:(nq + nkv) * d + nkv * dv].view(T, nkv, dv)
        if turned:
            q, k, v = plain.turn(q, pos, freq, stretch), plain.turn(k, pos, freq, stretch), plain.turn(v, pos, vfreq)
        tol = lambda ref: (3e-6 if dtype == torch.float32 else 2.0 ** -8) * float(ref.abs().max())
        assert (q_out.double().cpu().view(T, nq, d) - q).abs().max() <= tol(q)
        written = 0
        for i, (n, s) in enumerate(zip(lens, starts)):
            at = sum(lens[:i])
            kk, vv = rows_of(k_cache, table[i], page, s + n), rows_of(v_cache, table[i], page, s + n)
            assert (kk[s:] - k[at:at + n]).abs().max() <= tol(k) and (vv[s:] - v[at:at + n]).abs().max() <= tol(v)
            assert (kk[:s] == 3.0).all() and (vv[:s] == 3.0).all()
            written += n
        assert int((k_cache != 3.0).any(-1).sum()) <= written * nkv          # nothing else was touched
    o = torch.randn(T, nq * dv, generator=g).to(dtype)
    od = o.to(DEV)
    ops.turn_back(od, table_of(vfreq, 1.0), nq)
    ref = plain.turn(o.double().view(T, nq, dv), pos, vfreq, sign=-1.0)
    assert (od.double().cpu().view(T, nq, dv) - ref).abs().max() <= (3e-6 if dtype == torch.float32 else 2.0 ** -8) * float(ref.abs().max())


@pytest.mark.parametrize("pool,page,nkv,d,dv", [(1, 4, 1, 12, 10), (3, 4, 2, 64, 64), (12, 16, 1, 128, 64), (9, 8, 3, 6, 14), (64, 16, 2, 32, 32)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_means_of_blocks_of_cached_rows(pool, page, nkv, d, dv, dtype):
    """Blocks inside one portion, across portions, across pages and completed by single tokens (the input stage makes those):
    the mean of the rows as the cache holds them, and no other row of the pooled pages is touched."""
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(pool * page)
    n = 3 * pool + pool // 2 + 61
    tables = scattered_tables([n, n], page, 2 * -(-n // page) + 5, 1)
    ptables = torch.full(tables.shape, -1, dtype=torch.int32)
    rows = n // pool
    pages = torch.randperm(2 * -(-rows // page) + 3, generator=g)
    for i in range(2):
        for b in range(-(-rows // page)):
            ptables[i, b] = pages[i * -(-rows // page) + b]
    k_cache = torch.zeros(int(tables.max()) + 1, nkv, page, d, dtype=dtype, device=DEV)
    v_cache = torch.zeros(int(tables.max()) + 1, nkv, page, dv, dtype=dtype, device=DEV)
    pooled = ops.PooledRows(pool, torch.full((len(pages), nkv, page, d), 5.0, dtype=dtype, device=DEV),
                            torch.full((len(pages), nkv, page, dv), 5.0, dtype=dtype, device=DEV), ptables.to(DEV))
    nq = 2 * nkv
    wq, wk = torch.ones(nq * d), torch.ones(nkv * d)
    at = [0, 0]
    cuts = [[n - 40, 2] + [1] * 38, [2, pool, 7, n - 49 - pool] + [1] * 40]
    while any(c for c in cuts):
        parts = [(i, cuts[i].pop(0)) for i in (0, 1) if cuts[i]]
        step = FakeStep([m for _, m in parts], [at[i] for i, _ in parts])
        sel = [i for i, _ in parts]
        T = step.n_tokens
        qkv = torch.randn(T, nq * d + nkv * (d + dv), generator=g).to(dtype).to(DEV)
        q = torch.empty(T, nq * d, dtype=dtype, device=DEV)
        table = tables[sel].contiguous().to(DEV)
        p = ops.PooledRows(pool, pooled.k, pooled.v, ptables[sel].contiguous().to(DEV))
        if step.decode_only:
            ops.rows_norm_rope_cache(qkv, q, f32(wq), f32(wk), 1e-5, None, 0, None, step, table, k_cache, v_cache, nq, nkv, d, dv, pooled=p)
        else:
            with pytest.raises(ops.KernelError):
                ops.rows_norm_rope_cache(qkv, q, f32(wq), f32(wk), 1e-5, None, 0, None, step, table, k_cache, v_cache, nq, nkv, d, dv, pooled=p)
            ops.rows_norm_rope_cache(qkv, q, f32(wq), f32(wk), 1e-5, None, 0, None, step, table, k_cache, v_cache, nq, nkv, d, dv)
            ops.pool_means(k_cache, v_cache, p, step, table)
        for i, m in parts:
            at[i] += m
            done = at[i] // pool
            for cache, means in ((k_cache, pooled.k), (v_cache, pooled.v)):
                ref = plain.block_means(rows_of(cache, tables[i], page, at[i]), pool)
                got = rows_of(means, ptables[i], page, rows)
                assert (got[:done] - ref).abs().max() <= (1e-6 if dtype == torch.float32 else 2.0 ** -8) * float(ref.abs().max()) if done else True
                assert (got[done:] == 5.0).all()
    assert at == [n, n]


def pooled_case(nq, nkv, d, dv, size, pool, page, lens, starts, dtype, seed, loud=()):
    """Caches, tables and queries of a batch, with every sequence's keys and values in place, and the plain result.  `loud`:
    (sequence, position, what): the query at that position is made to point at one key ("token", j) or pooled block
    ("block", b) with a score far above the others, whether the position may see it or not."""
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(seed)
    totals = [s + n for s, n in zip(starts, lens)]
    tables = scattered_tables(totals, page, sum(-(-n // page) for n in totals) + 7, seed)
    rows = [n // pool for n in totals]
    ptables = scattered_tables(rows, page, sum(-(-n // page) for n in rows) + 3, seed + 1)
    wide = max(tables.shape[1], ptables.shape[1])
    grow = lambda t: torch.cat([t, torch.full((t.shape[0], wide - t.shape[1]), -1, dtype=torch.int32)], dim=1)
    tables, ptables = grow(tables), grow(ptables)
    mk = lambda n, s: torch.zeros(n, nkv, page, s, dtype=dtype)
    n_pages, n_rows = int(tables.max()) + 1, max(int(ptables.max()) + 1, 1)
    k_cache, v_cache, pk, pv = mk(n_pages, d), mk(n_pages, dv), mk(n_rows, d), mk(n_rows, dv)
    q = torch.randn(sum(lens), nq * d, generator=g).to(dtype)
    keys, values = [], []
    for i, n in enumerate(totals):
        k, v = torch.randn(n, nkv, d, generator=g).to(dtype), torch.randn(n, nkv, dv, generator=g).to(dtype)
        for s_, pos, (kind, j) in loud:
            if s_ == i and pos < n:
                k[j * pool:(j + 1) * pool] = (k[j * pool:(j + 1) * pool].float() * 2 + 1.5 * torch.randn(1, nkv, d, generator=g)).to(dtype) if kind == "block" else k[j * pool:(j + 1) * pool]
        keys.append(k); values.append(v)
        for j in range(n):
            k_cache[tables[i, j // page], :, j % page] = k[j]
            v_cache[tables[i, j // page], :, j % page] = v[j]
        kb, vb = plain.block_means(k.double(), pool).to(dtype), plain.block_means(v.double(), pool).to(dtype)
        for b in range(kb.shape[0]):
            pk[ptables[i, b // page], :, b % page] = kb[b]
            pv[ptables[i, b // page], :, b % page] = vb[b]
    for s_, pos, (kind, j) in loud:
        if starts[s_] <= pos < totals[s_]:
            t = sum(lens[:s_]) + pos - starts[s_]
            k = keys[s_].float()
            target = k[j] if kind == "token" else k[j * pool:(j + 1) * pool].mean(0)
            target = target / target.norm(dim=-1, keepdim=True) * math.sqrt(d)
            q[t] = (3.0 * target.repeat_interleave(nq // nkv, dim=0)).reshape(-1).to(dtype)
    # a window lets earlier pages go: they are no longer in the tables when the step runs
    tables = tables.clone()
    for i, s in enumerate(starts):
        for b in range(max(0, s - max(size, pool) + 1) // page):
            tables[i, b] = -1
    scale = 1.0 / math.sqrt(d)
    ref = torch.zeros(sum(lens), nq, dv, dtype=torch.float64)
    for i, (n, s) in enumerate(zip(lens, starts)):
        at = sum(lens[:i])
        k, v = keys[i].double(), values[i].double()
        kb, vb = plain.block_means(k, pool).to(dtype).double(), plain.block_means(v, pool).to(dtype).double()
        tok, blk = plain.visible(s + n, size, pool)
        seen = torch.cat([tok, blk], dim=1)[s:]
        for h in range(nq):
            kv = h // (nq // nkv)
            sc = q[at:at + n].double().view(n, nq, d)[:, h] @ torch.cat([k[:, kv], kb[:, kv]]).T * scale
            ref[at:at + n, h] = torch.softmax(sc.masked_fill(~seen, float("-inf")), dim=-1) @ torch.cat([v[:, kv], vb[:, kv]])
    pooled = ops.PooledRows(pool, pk.to(DEV), pv.to(DEV), ptables.to(DEV))
    return q.to(DEV), k_cache.to(DEV), v_cache.to(DEV), pooled, tables.to(DEV), scale, ref


def run_pooled(case, lens, starts, nq, nkv, d, dv, size, turn=None):
    from inferloop_b200.csrc import ops
    from inferloop_b200.parts.base import Workspace
    q, kc, vc, pooled, tables, scale, ref = case
    step = FakeStep(lens, starts)
    out = torch.full((sum(lens), nq * dv), 9.0, dtype=q.dtype, device=DEV)
    ops.attention(q, out, kc, vc, step, tables, size, scale, nq, nkv, d, workspace=Workspace(torch.device(DEV)), dv=dv, pooled=pooled, turn=turn)
    ops.check_device_errors()
    return out.double().cpu().view(sum(lens), nq, dv)


GEOMETRIES = [(5, 1, 12, 10, 7, 3, 4), (4, 4, 6, 14, 5, 9, 4), (8, 2, 64, 64, 50, 8, 16), (4, 1, 128, 64, 20, 4, 16), (2, 2, 128, 128, 33, 1, 16),
              (32, 1, 64, 64, 70, 5, 32), (20, 1, 128, 64, 40, 24, 16), (1, 1, 64, 64, 1, 2, 16), (6, 3, 128, 128, 200, 16, 64)]


@pytest.mark.parametrize("nq,nkv,d,dv,size,pool,page", GEOMETRIES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", ["whole", "portions", "single", "mixed", "far"])
def test_attention_over_a_window_and_pooled_blocks(nq, nkv, d, dv, size, pool, page, dtype, shape):
    """Portions from the start and behind cached tokens, single tokens, both in one batch, and far into a sequence (hundreds of
    pooled rows), with and without turning the output back.  Queries point at single keys and blocks just inside and just
    outside what they may see."""
    from inferloop_b200.csrc import ops
    lens, starts = {"whole": ([150, 3], [0, 0]), "portions": ([130, 2, 40], [77, 150, 3]), "single": ([1, 1, 1, 1], [0, size, 3 * pool + size, 260]),
                    "mixed": ([1, 45, 1, 2], [301, 140, 0, 90]), "far": ([30, 1], [900 + 300 * min(pool, 4), 2000])}[shape]
    loud = []
    for i, (n, s) in enumerate(zip(lens, starts)):
        for pos in sorted({s, s + n // 2, s + n - 1}):
            first = max(0, pos - size + 1)
            b = first // pool
            picks = [("token", first)] + ([("token", first - 1)] if first else []) + ([("block", b - 1)] if b else []) + \
                    ([("block", b)] if (b + 1) * pool <= s + n else [])
            loud.append((i, pos, picks[(pos + i) % len(picks)]))
    case = pooled_case(nq, nkv, d, dv, size, pool, page, lens, starts, dtype, nq * d + size + len(shape), loud)
    q, kc, vc, pooled, tables, scale, ref = case
    tol = (2e-5 if dtype == torch.float32 else 1.2e-2) * float(ref.abs().max())
    for force in ((0, 1, 2) if dtype == torch.bfloat16 else (0,)):
        ops.TC_ATTENTION_ROW_BLOCKS = force
        try:
            out = run_pooled(case, lens, starts, nq, nkv, d, dv, size)
            err = (out - ref).abs().max()
            assert err <= tol, f"row blocks {force}: {float(err):.3e} of {float(ref.abs().max()):.3e}"
            if dv % 2 == 0:
                pos = FakeStep(lens, starts).positions.cpu()
                freq, _ = plain.frequencies(300.0, dv)
                ang = pos.double()[:, None] * freq
                out = run_pooled(case, lens, starts, nq, nkv, d, dv, size, f32(torch.stack([torch.cos(ang), torch.sin(ang)], dim=-1)))
                assert (out - plain.turn(ref, pos, freq, sign=-1.0)).abs().max() <= 1.5 * tol
        finally:
            ops.TC_ATTENTION_ROW_BLOCKS = 0
    if dtype == torch.bfloat16:          # the exact kernel on the same bfloat16 inputs
        ops.TC_ATTENTION_ENABLED = False
        try:
            assert (run_pooled(case, lens, starts, nq, nkv, d, dv, size) - ref).abs().max() <= tol
        finally:
            ops.TC_ATTENTION_ENABLED = True


@pytest.mark.parametrize("size,pool", [(50, 8), (20, 3), (1, 1)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_every_edge_of_a_window_and_of_a_block(size, pool, dtype):
    """One position after another as a single token whose query points at the key at the window's edge, at the one before it,
    at the last visible block and at the next one: what is seen dominates, what is not seen does not."""
    nq, nkv, d, dv, page = 8, 2, 64, 64, 16
    for pos in list(range(size - 1, size + 2 * pool + 3)) + [191, 192, 193]:
        first = max(0, pos - size + 1)
        b = first // pool
        for what in [("token", first)] + ([("token", first - 1)] if first else []) + ([("block", b - 1)] if b else []) + \
                ([("block", b)] if (b + 1) * pool <= pos + 1 else []):
            case = pooled_case(nq, nkv, d, dv, size, pool, page, [1], [pos], dtype, pos * 7 + size, [(0, pos, what)])
            ref = case[-1]
            out = run_pooled(case, [1], [pos], nq, nkv, d, dv, size)
            assert (out - ref).abs().max() <= (2e-5 if dtype == torch.float32 else 1.2e-2) * float(ref.abs().max()), (pos, what)


DELTA = [(3, 10, 10), (1, 20, 20), (2, 64, 64), (2, 128, 128), (1, 200, 40), (2, 32, 96), (1, 1, 1), (3, 48, 48), (4, 128, 64)]


@pytest.mark.parametrize("heads,d,dv", DELTA)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_delta_rule_whole_and_in_portions(heads, d, dv, dtype):
    """Two sequences against the token-by-token recurrence in 64-bit: whole (chunks side by side where they apply), in portions
    down to two tokens and token by token through the state slot; decays from one token to thousands, removal rates from
    none to all, a first token that stands out behind the slow channels, a key of zero."""
    from inferloop_b200.csrc import ops
    from inferloop_b200.parts.base import Workspace
    g = torch.Generator().manual_seed(heads * d + dv)
    lens = [330, 45]
    wk, wv = heads * d, heads * dv
    log_decay, unit_eps = 0.7, 1e-4
    w0, ab = torch.linspace(-9.0, 3.0, wk), torch.linspace(-6.0, 5.0, wk).flip(0)
    proj, low, ref = [], [], []
    for n in lens:
        p = torch.randn(n, 3 * wk + wv + 6, generator=g)
        p[0, 3 * wk:3 * wk + wv] *= 20.0
        p[7, wk:2 * wk] = 0.0
        l = torch.randn(n, wk, generator=g)
        p = p.to(dtype)
        x = p.double()
        heads_of = lambda t, s: t.reshape(n, heads, s)
        decay = torch.exp(-log_decay * torch.sigmoid(l.double() + w0.double()))
        removal = torch.sigmoid(x[:, 2 * wk:3 * wk] + ab.double())
        keep = plain.UNIT_EPS
        plain.UNIT_EPS = unit_eps
        try:
            o, S = plain.delta_rule(heads_of(decay, d), heads_of(removal, d), heads_of(x[:, wk:2 * wk], d), heads_of(x[:, 3 * wk:3 * wk + wv], dv),
                                    heads_of(x[:, :wk], d))
        finally:
            plain.UNIT_EPS = keep
        proj.append(p); low.append(l); ref.append((o.reshape(n, wv), S))
    ws = Workspace(torch.device(DEV))
    for mode, cuts in (("whole", [[330], [45]]), ("portions", [[1, 2, 130, 17, 2, 150, 28], [40, 5]]), ("single", [[290] + [1] * 40, [5] + [1] * 40])):
        state = torch.full((3, heads, d, dv), 5.0, dtype=torch.float32, device=DEV)
        state[0].zero_(); state[2].zero_()
        at = [0, 0]
        for k in range(max(len(c) for c in cuts)):
            parts = [(s, at[s], at[s] + cuts[s][k]) for s in (0, 1) if k < len(cuts[s])]
            step = FakeStep([b - a for _, a, b in parts], [a for _, a, _ in parts], [2 if s == 0 else 0 for s, _, _ in parts])
            x = torch.cat([proj[s][a:b] for s, a, b in parts]).to(DEV)
            l = f32(torch.cat([low[s][a:b] for s, a, b in parts]))
            y = torch.empty(x.shape[0], wv, dtype=torch.float32, device=DEV)
            ops.delta_scan(x, 0, wk, 3 * wk, 2 * wk, l, f32(w0), f32(ab), log_decay, unit_eps, state, y, step, heads, d, dv, workspace=ws)
            want = torch.cat([ref[s][0][a:b] for s, a, b in parts])
            for i, (s, a, b) in enumerate(parts):            # (a sequence's own size: the first token of each stands out)
                lo = sum(q_ - p_ for _, p_, q_ in parts[:i])
                got = y[lo:lo + b - a].double().cpu()
                err = (got - ref[s][0][a:b]).abs().max() / ref[s][0].abs().max()
                assert err < 2e-5, f"{mode} step {k}: {float(err):.3e}"
                at[s] = b
        for s, slot in ((0, 2), (1, 0)):
            err = (state[slot].double().cpu() - ref[s][1]).abs().max() / ref[s][1].abs().max()
            assert err < 2e-5, f"{mode} final state: {float(err):.3e}"
        assert float(state[1].min()) == 5.0 and float(state[1].max()) == 5.0
    # a dummy row (no slot) starts from zero and stores nothing
    before = state.clone()
    step = FakeStep([1], [0], [-1])
    y = torch.empty(1, wv, dtype=torch.float32, device=DEV)
    ops.delta_scan(proj[1][:1].to(DEV), 0, wk, 3 * wk, 2 * wk, f32(low[1][:1]), f32(w0), f32(ab), log_decay, unit_eps, state, y, step, heads, d, dv, workspace=ws)
    assert torch.equal(state, before)
    assert (y.double().cpu() - ref[1][0][:1]).abs().max() <= 2e-5 * ref[1][0].abs().max()


@pytest.mark.parametrize("heads,d,dv,rank", [(2, 64, 64, 24), (3, 128, 128, 5), (1, 128, 64, 200), (4, 10, 12, 1), (2, 48, 48, 16), (5, 100, 4, 33)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_single_tokens_of_the_delta_rule_in_one_launch(heads, d, dv, rank, dtype):
    """The low-rank map, decay, recurrence, norm of each head and gate of several sequences' single tokens, step after step, from
    states that are not zero; a dummy row beside them; slots of others are left alone."""
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(heads * d + rank)
    wk, wv = heads * d, heads * dv
    pad = -rank % 8
    log_decay, unit_eps, eps = 0.6, 1e-6, 1e-5
    w2 = torch.zeros(wk, rank + pad)
    w2[:, :rank] = torch.randn(wk, rank, generator=g) / math.sqrt(rank)
    w2 = w2.to(dtype)
    w0, ab, norm = torch.linspace(-9.0, 2.0, wk), torch.linspace(-3.0, 3.0, wk).flip(0), 1 + 0.2 * torch.randn(wv, generator=g)
    state = torch.randn(6, heads, d, dv, generator=g)
    ref_state = {0: state[4].double(), 1: state[1].double(), 3: state[5].double()}
    dev = f32(state)
    slots = [4, 1, -1, 5]
    n = len(slots)
    for _ in range(5):
        proj = torch.randn(n, 3 * wk + 2 * wv + rank + pad, generator=g).to(dtype)
        out = torch.full((n, wv), 9.0, dtype=dtype, device=DEV)
        step = FakeStep([1] * n, [3, 7, 0, 9], slots)
        ops.delta_step(proj.to(DEV), 0, wk, 3 * wk, 2 * wk, 3 * wk + wv, 3 * wk + 2 * wv, rank, w2.to(DEV), f32(w0), f32(ab), log_decay, unit_eps, f32(norm),
                       eps, dev, out, step, heads, d, dv)
        x = proj.double()
        decay = torch.exp(-log_decay * torch.sigmoid(torch.tanh(x[:, 3 * wk + 2 * wv:3 * wk + 2 * wv + rank]) @ w2.double()[:, :rank].T + w0.double()))
        removal = torch.sigmoid(x[:, 2 * wk:3 * wk] + ab.double())
        for i in range(n):
            one = lambda t, s: t[i].reshape(1, heads, s)
            o, S = plain.delta_rule(one(decay, d), one(removal, d), one(x[:, wk:2 * wk], d), one(x[:, 3 * wk:3 * wk + wv], dv), one(x[:, :wk], d), ref_state.get(i))
            want = plain.rms(o, eps).reshape(wv) * norm.double() * torch.sigmoid(x[i, 3 * wk + wv:3 * wk + 2 * wv])
            assert (out[i].double().cpu() - want).abs().max() <= (2e-5 if dtype == torch.float32 else 2.0 ** -7) * want.abs().max()
            if i in ref_state:
                ref_state[i] = S
    for i, s in ((0, 4), (1, 1), (3, 5)):
        assert (dev[s].double().cpu() - ref_state[i]).abs().max() <= 2e-5 * ref_state[i].abs().max()
    for s in (0, 2, 3):
        assert torch.equal(dev[s].cpu(), state[s])
