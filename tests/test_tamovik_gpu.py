"""The Tamovik decoder through the engine, and each of its mechanisms alone (GPU), against the plain 64-bit statement in
plain_tamovik.py.  The configurations are in tamovik_cases.py: K (odd sizes, exact kernels, a layer without feed-forward), L
(the tensor-core kernels' sizes), M (everything plural is one), N (no latent layer, no chunks, no second table), P (rows of more
than 512 elements, a state of 256 rows, groups of twenty heads)."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_tamovik as plain
import tamovik_cases as cases
from helpers import ROOT, Trace, assert_close, random_tokens, run_trace_inprocess

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ENGINE_CASES = [(n, d) for n in ("K", "L", "M", "N", "P") for d in ("float32", "bfloat16")]
# bfloat16: the norm on a sublayer's output divides by that output's own size, so a rounding reaches the stream undamped, and
# where a small output is the difference of large terms it is magnified.  Against the 64-bit statement with the same weights
# the logits of a position differ, root-mean-square, by 0.2 % of the largest logit at the median position, by more than 1 % at a
# few in a hundred.  A fault (a wrong key, a lost state) costs tens of per cent.  32-bit runs have no such allowance.
BF16_MOST, BF16_ALL = 0.01, 0.04


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return str(tmp_path_factory.mktemp("tamovik"))


def stored(dtype):
    return torch.bfloat16 if dtype == "bfloat16" else torch.float32


def runner_for(root, name, dtype, pages=64, requests=4, page=None):
    from inferloop_b200.engine import ModelRunner
    _, _, page_size = cases.CASES[name]
    return ModelRunner.from_folder(cases.folder(root, name, stored(dtype)), dtype=dtype, device=DEV,
                                   page_size=page or page_size, num_pages=pages, max_requests=requests)


_TOKENS = {}


def tokens_for(root, name, dtype, n, seed):
    key = (name, dtype, n, seed)
    if key not in _TOKENS:
        model = cases.plain_model(root, name, stored(dtype))
        _TOKENS[key] = cases.decided_tokens(model, n, cases.CASES[name][0]["vocab"], seed, 4e-2 if dtype == "bfloat16" else 1e-4)
    return _TOKENS[key]


def reference(root, name, dtype, tokens):
    return cases.plain_model(root, name, stored(dtype)).forward(tokens)


def check_rows(got, ref, dtype, what):
    """Rows of logits (or of the stream) against the plain statement's."""
    got, ref = got.double().cpu(), ref.double()
    assert got.shape == ref.shape and torch.isfinite(got).all(), what
    if dtype == "float32":
        assert_close(got, ref, dtype, what)
        return
    err = (got - ref).pow(2).mean(-1).sqrt() / float(ref.abs().max())
    worst = torch.topk(err, min(5, len(err)))
    over = int((err > BF16_MOST).sum())
    assert float(worst.values[0]) <= BF16_ALL and over <= max(1, len(err) // 10), \
        f"{what}: {over} of {len(err)} rows over {BF16_MOST}, worst {worst.values.tolist()} at {worst.indices.tolist()}"


def check_trace(outputs, trace, ref, dtype, what):
    rows = [(s, i, rid, pos) for s, rr in trace.rows.items() for i, (rid, pos) in enumerate(rr)]
    check_rows(torch.stack([torch.from_numpy(outputs[s][i]) for s, i, _, _ in rows]), torch.stack([ref[rid][pos] for _, _, rid, pos in rows]), dtype, what)


# ------------------------------------------------------------------------------ the engine
@pytest.mark.parametrize("name,dtype", ENGINE_CASES)
def test_whole_prompt_and_every_layer(root, name, dtype):
    """One prompt in one step: the residual stream after every layer, and all logits."""
    from inferloop_b200.engine import StepEntry
    r = runner_for(root, name, dtype)
    toks = tokens_for(root, name, dtype, 45, 1)
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
        check_rows(g, w, dtype, f"{name} layer {i}")
    check_rows(logits, ref, dtype, f"{name} logits")


@pytest.mark.parametrize("name,dtype", ENGINE_CASES)
def test_prefill_against_token_by_token_and_portions(root, name, dtype):
    """The same sequence token by token from the first token on, and in portions of changing size down to two tokens with
    the last tokens one by one: over the borders of chunks and pages of every case."""
    toks = tokens_for(root, name, dtype, 90, 2)
    ref = {"a": reference(root, name, dtype, toks)}
    r = runner_for(root, name, dtype, pages=80)
    t = Trace()
    for i, tok in enumerate(toks[:75]):
        t.step([("a", [tok], [0])], end=["a"] if i == 74 else [])
    check_trace(run_trace_inprocess(r, t), t, ref, dtype, f"{name} token by token")
    t = Trace()
    at = 0
    for n in (2, 5, 3, 17, 2, 9, 20, 1, 2, 7):
        t.step([("a", toks[at:at + n], list(range(n)))])
        at += n
    while at < len(toks):
        t.step([("a", toks[at:at + 1], [0])], end=["a"] if at == len(toks) - 1 else [])
        at += 1
    check_trace(run_trace_inprocess(r, t), t, ref, dtype, f"{name} portions")
    r.cache.check()
    assert all(n == g.pool.num_pages for g, n in zip(r.cache.groups, r.cache.free_pages().values()))


@pytest.mark.parametrize("page", [32, 64, 128])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_larger_pages(root, page, dtype):
    """The tensor-core sizes over pages that chunks end inside of, two requests side by side."""
    toks = {k: tokens_for(root, "L", dtype, n, 20 + n) for k, n in (("a", 90), ("b", 64))}
    ref = {k: reference(root, "L", dtype, v) for k, v in toks.items()}
    r = runner_for(root, "L", dtype, pages=2 * -(-90 // page), page=page)
    t = Trace()
    t.step([("a", toks["a"][:57], list(range(57))), ("b", toks["b"][:2], [0, 1])])
    t.step([("a", toks["a"][57:70], [0, 12]), ("b", toks["b"][2:50], list(range(48)))])
    for i in range(14):
        t.step([("a", toks["a"][70 + i:71 + i], [0]), ("b", toks["b"][50 + i:51 + i], [0])], end=["b"] if i == 13 else [])
    t.step([("a", toks["a"][84:], list(range(6)))], end=["a"])
    check_trace(run_trace_inprocess(r, t), t, ref, dtype, f"pages of {page}")


@pytest.mark.parametrize("name,dtype", ENGINE_CASES)
def test_mixed_batches_with_pages_and_slots_used_again(root, name, dtype):
    """Up to four live requests of unequal length, portions beside single tokens, four state slots for seven requests and a
    pool that cannot hold all of them: what ends gives its pages and its slot (state, normaliser, maximum, the convolution's
    inputs, the previous token) to the next.  Every row equals the request alone."""
    lens = {"a": 37, "b": 5, "c": 64, "d": 21, "e": 50, "f": 2, "g": 33}
    toks = {k: tokens_for(root, name, dtype, n, 10 + i) for i, (k, n) in enumerate(lens.items())}
    ref = {k: reference(root, name, dtype, v) for k, v in toks.items()}
    page = cases.CASES[name][2]
    pages = -(-64 // page) + -(-50 // page) + -(-37 // page) + -(-33 // page)
    r = runner_for(root, name, dtype, pages=pages, requests=4)
    t = Trace()
    cursor = {k: 0 for k in lens}
    waiting, live = list(lens), []
    portion = {"a": [2, 16, 3], "b": [5], "c": [31, 2, 20], "d": [8, 8], "e": [3, 40], "f": [2], "g": [30]}
    step = 0
    while waiting or live:
        while waiting and len(live) < 4:
            if sum(-(-lens[k] // page) for k in live + [waiting[0]]) > pages:
                break
            live.append(waiting.pop(0))
        entries, ended = [], []
        for k in live:
            n = min(portion[k].pop(0) if portion[k] else 1, lens[k] - cursor[k])
            entries.append((k, toks[k][cursor[k]:cursor[k] + n], sorted({0, n - 1})))
            cursor[k] += n
            if cursor[k] == lens[k]:
                ended.append(k)
        t.step(entries, end=ended)
        live = [k for k in live if k not in ended]
        step += 1
        assert step < 400
    check_trace(run_trace_inprocess(r, t), t, ref, dtype, f"{name} mixed")
    info = r.cache.inspect()
    assert info["begun"] == len(lens) and info["live_requests"] == 0
    assert any(g["reuses"] > 0 for g in info["groups"]), "no page was used again"
    r.cache.check()


@pytest.mark.parametrize("name,dtype", [("K", "float32"), ("L", "bfloat16"), ("M", "float32"), ("N", "bfloat16")])
def test_long_decoding_through_recorded_graphs(root, name, dtype):
    """A short prompt, then 140 single tokens (recorded decode graphs after the first), over many chunks' borders, with the slow
    heads of the memory still carrying the prompt at the end."""
    toks = tokens_for(root, name, dtype, 160, 3)
    ref = {"a": reference(root, name, dtype, toks)}
    r = runner_for(root, name, dtype, pages=-(-170 // cases.CASES[name][2]))
    t = Trace()
    t.step([("a", toks[:20], [19])])
    for i in range(20, len(toks)):
        t.step([("a", [toks[i]], [0])], end=["a"] if i == len(toks) - 1 else [])
    check_trace(run_trace_inprocess(r, t), t, ref, dtype, f"{name} long decoding")
    assert r.graphs is not None and r.graphs.whole and r.graphs.replays > 100


@pytest.mark.parametrize("name,dtype", [("K", "float32"), ("L", "float32"), ("L", "bfloat16"), ("M", "float32"), ("N", "float32"), ("N", "bfloat16")])
def test_a_long_prompt_whole_and_in_portions(root, name, dtype):
    """700 tokens in one step (the memory runs in chunks of 64 on bfloat16) against the same prompt in portions of 128 (chunks
    again, other borders), 100 and 11 (token by token): the logits at a position do not depend on the cut."""
    from inferloop_b200.engine import StepEntry
    toks = random_tokens(700, cases.CASES[name][0]["vocab"], 77)
    want = list(range(5, 700, 10)) + [699]
    r = runner_for(root, name, dtype, pages=-(-700 // cases.CASES[name][2]) + 2)
    whole = r.step([StepEntry("w", toks, want)]).float().cpu().clone()
    r.end("w")
    if dtype == "float32":
        model = cases.plain_model(root, name, stored(dtype))
        if model.least_margin(toks) > 1e-4:
            assert_close(whole, model.forward(toks)[want], dtype, f"{name} 700 tokens whole")
    for portion in (128, 100, 11):
        rows = []
        for at in range(0, 700, portion):
            part = toks[at:at + portion]
            out = r.step([StepEntry("p", part, [w - at for w in want if at <= w < at + len(part)])])
            rows.append(out.float().cpu().clone())
        r.end("p")
        rows = torch.cat(rows)
        if dtype == "float32":
            err = (rows.double() - whole.double()).abs().max()
            assert err <= 3e-5 * whole.abs().max(), f"{name} portions of {portion}: {float(err):.3e}"
        else:
            # (random tokens: a routing decision may be close; all but a few rows agree within rounding)
            err = (rows.double() - whole.double()).pow(2).mean(-1).sqrt() / float(whole.abs().max())
            assert int((err > BF16_MOST).sum()) <= len(want) // 10, f"{name} portions of {portion}: {sorted(err.tolist())[-10:]}"


@pytest.mark.parametrize("name,dtype", [("K", "float32"), ("L", "bfloat16"), ("M", "float32")])
def test_greedy_generation_through_the_entry_point(root, name, dtype):
    from inferloop_b200 import Engine, SamplingParams
    _, _, page = cases.CASES[name]
    model = cases.plain_model(root, name, stored(dtype))
    prompts = [tokens_for(root, name, dtype, n, 30 + n) for n in (3, 12, 31, 64)]
    engine = Engine(cases.folder(root, name, stored(dtype)), dtype=dtype, block_size=page, num_gpu_blocks_override=96,
                    max_num_seqs=4, prefill_chunk_tokens=32, max_num_batched_tokens=40)
    new = 12
    got = engine.generate(prompts, SamplingParams(), max_new_tokens=new)
    for p, g in zip(prompts, got):
        assert len(g) == new
        ref = model.forward(list(p) + list(g))[len(p) - 1:-1]
        bound = (2 * BF16_MOST if dtype == "bfloat16" else 1e-5) * float(ref.abs().max())
        for i, tok in enumerate(g):        # teacher-forced: every chosen token is the best one within the bound
            assert ref[i, tok] >= ref[i].max() - 2 * bound
    info = engine.inspect()
    assert info["running"] == 0 and all(g["free"] == g["total"] for g in info["cache"]["groups"])


def test_the_command_line_generates_from_a_tamovik_folder(root):
    name, dtype = "M", "float32"
    prompt = tokens_for(root, name, dtype, 9, 41)
    out = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "infer"), "generate", cases.folder(root, name, stored(dtype)),
                          "--tokens", ",".join(map(str, prompt)), "--max-new-tokens", "6", "--dtype", dtype, "--block-size", "16",
                          "--num-gpu-blocks-override", "8"], capture_output=True, text=True, timeout=900)
    assert out.returncode == 0, out.stderr
    got = json.loads(out.stdout.strip().splitlines()[-1])["tokens"]
    ref = cases.plain_model(root, name, stored(dtype)).forward(list(prompt) + got)[len(prompt) - 1:-1]
    for i, tok in enumerate(got):
        assert ref[i, tok] >= ref[i].max() - 2e-5 * float(ref.abs().max())


def test_the_trace_program_replays_a_tamovik_folder(root, tmp_path):
    name, dtype = "K", "float32"
    toks = {"x": tokens_for(root, name, dtype, 40, 5), "y": tokens_for(root, name, dtype, 9, 6)}
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
    check_trace(out, t, ref, dtype, "trace program")


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
        self.slots = i32(list(range(len(lens))) if slots is None else slots)
        self.h_kv_len = [s + n for n, s in zip(lens, starts)]
        self.max_kv_len = max(self.h_kv_len)
        self.position_tables = {}


def f32(t):
    return t.float().to(DEV).contiguous()


def workspace():
    from inferloop_b200.parts import Workspace
    return Workspace(torch.device(DEV))


def scattered_tables(lens, page, pages, seed):
    """Block tables whose pages lie anywhere in the pool: [seqs, max_blocks] int32, -1 where nothing is held."""
    order = torch.randperm(pages, generator=torch.Generator().manual_seed(seed)).tolist()
    table = torch.full((len(lens), max(-(-n // page) for n in lens) + 3), -1, dtype=torch.int32)
    for i, n in enumerate(lens):
        for b in range(-(-n // page)):
            table[i, b] = order.pop()
    return table


def rows_of(cache, table, page, n):
    """[n, heads, size] rows 0 .. n - 1 of a sequence from the pages, in 64-bit."""
    return torch.stack([cache[table[j // page], :, j % page] for j in range(n)]).double().cpu()


def put_rows(cache, table, page, rows):
    for j in range(rows.shape[0]):
        cache[table[j // page], :, j % page] = rows[j].to(cache.dtype).to(cache.device)


# (nq, nkv, d, page, chunk): the exact kernel, the kernels of head size 32 and 96, and those of 64 and 128
CHUNKED = [(6, 2, 12, 4, 5), (3, 1, 32, 16, 24), (4, 2, 96, 16, 70), (8, 2, 64, 16, 40), (4, 1, 128, 16, 100), (2, 2, 64, 64, 64), (5, 1, 128, 32, 1),
           (16, 1, 64, 128, 333), (4, 4, 20, 8, 1000)]


@pytest.mark.parametrize("nq,nkv,d,page,chunk", CHUNKED)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_attention_inside_aligned_chunks(nq, nkv, d, page, chunk, dtype):
    """Every kernel that takes a chunk: a long portion, short portions and single tokens, alone and mixed, at chunk borders, one
    before and one behind them.  The last key of every chunk and the first of the next stand out for every query: one that is
    seen by mistake, or missed, changes the output altogether."""
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(nq * d + chunk)
    n = 420
    u = torch.randn(d, generator=g)
    u = u / u.norm() * d ** 0.25 * 2.6
    k = torch.randn(n, nkv, d, generator=g) * 0.6
    v = torch.randn(n, nkv, d, generator=g)
    for b in range(chunk, n, chunk):
        k[b - 1] += u
        k[b] += u
    k, v = k.to(dtype), v.to(dtype)
    scale = d ** -0.5
    full = (torch.randn(n, nq, d, generator=g) + u).to(dtype)
    ref = plain.softmax_attention(full.double(), k.double(), v.double(), scale, plain.same_chunk(n, chunk))
    ws = workspace()
    pages = 4 * -(-n // page) + 4
    edges = sorted({min(max(p, 0), n - 1) for b in (chunk, 2 * chunk, n // chunk * chunk) for p in (b - 1, b, b + 1)} | {0, n - 1})
    batches = [[(0, n)], [(0, 2), (n - 3, 3)], [(p, 1) for p in edges], [(p, 1) for p in edges[:3]] + [(max(edges[-2] - 30, 0), 31)],
               [(max(0, chunk - 3), min(9, n - max(0, chunk - 3))), (5, 150)]]
    for spans in batches:
        starts, lens = [s for s, _ in spans], [m for _, m in spans]
        step = FakeStep(lens, starts)
        ends = [s + m for s, m in spans]
        tables = scattered_tables(ends, page, len(spans) * -(-n // page) + 4, len(spans))
        k_cache = torch.zeros(int(len(spans) * -(-n // page) + 4), nkv, page, d, dtype=dtype, device=DEV)
        v_cache = torch.zeros_like(k_cache)
        for i, e in enumerate(ends):
            put_rows(k_cache, tables[i], page, k[:e])
            put_rows(v_cache, tables[i], page, v[:e])
            first = (starts[i] // chunk * chunk) // page        # pages that nobody in this step reads are gone
            tables[i, :first] = -1
        q = torch.cat([full[s:s + m] for s, m in spans]).reshape(-1, nq * d).to(DEV).contiguous()
        out = torch.empty_like(q)
        ops.attention(q, out, k_cache, v_cache, step, tables.to(DEV), -chunk, scale, nq, nkv, d, workspace=ws)
        want = torch.cat([ref[s:s + m] for s, m in spans]).reshape(-1, nq * d)
        tol = 2e-5 if dtype == torch.float32 else 2e-2
        assert (out.double().cpu() - want).abs().max() <= tol * float(v.double().abs().max()), (spans[:3], float((out.double().cpu() - want).abs().max()))
    ops.check_device_errors()


@pytest.mark.parametrize("switch", ["DECODE_CLUSTER_ENABLED", "TC_ATTENTION_ENABLED", "FLASH_ENABLED", "MIXED_SPLIT_ENABLED"])
def test_chunks_on_the_other_kernels(switch, monkeypatch):
    """The same geometry on the kernels that another one usually stands in front of."""
    from inferloop_b200.csrc import ops
    monkeypatch.setattr(ops, switch, False)
    test_attention_inside_aligned_chunks(8, 2, 64, 16, 40, torch.bfloat16)
    test_attention_inside_aligned_chunks(4, 1, 128, 16, 300, torch.bfloat16)


@pytest.mark.parametrize("nq,nkv,d,dv,taps,rd,page", [(6, 2, 12, 12, 5, 0, 4), (1, 1, 7, 7, 1, 0, 8), (8, 2, 64, 64, 4, 0, 16), (2, 1, 128, 128, 3, 64, 16),
                                                      (3, 3, 40, 24, 2, 16, 8), (40, 8, 128, 128, 4, 0, 64)])
@pytest.mark.parametrize("keys", [True, False])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_convolutions_before_norms_over_whole_rows(nq, nkv, d, dv, taps, rd, page, keys, dtype):
    """Three sequences over four steps (a portion, two tokens, single tokens, a portion beside single tokens), so that the inputs
    ahead of a step come from the state slots; values that are the convolved keys, and values of their own; with and without a
    rotation; a padding row without a slot."""
    from inferloop_b200.csrc import ops
    if keys and dv != d:
        pytest.skip("values that are keys have the keys' size")
    g = torch.Generator().manual_seed(nq * d + taps)
    n, seqs, width = 30, 3, (nq + nkv) * d
    size = torch.logspace(-0.5, 0.5, nq + nkv).repeat_interleave(d)
    extra = 0 if keys else nkv * dv
    pad = -(width + extra) % 8 + 8
    raw = [(torch.randn(n, width + extra + pad, generator=g) * torch.cat([size, torch.ones(extra + pad)])).to(dtype) for _ in range(seqs)]
    cw = torch.randn(width, taps, generator=g)
    wq, wk = 1 + 0.3 * torch.randn(nq * d, generator=g), 1 + 0.3 * torch.randn(nkv * d, generator=g)
    freq, _ = plain.frequencies({"base": 50.0, "dims": max(rd, 2)})
    ref = []
    for x in raw:
        x = x.double()
        u = plain.short_conv(x[:, :width], cw.double())
        q, k = plain.norm(u[:, :nq * d], wq.double(), 1e-4).view(n, nq, d), plain.norm(u[:, nq * d:], wk.double(), 1e-4).view(n, nkv, d)
        v = u[:, nq * d:].view(n, nkv, d) if keys else x[:, width:width + extra].view(n, nkv, dv)
        if rd:
            rot = {"base": 50.0, "dims": rd}
            q, k = plain.turn(q, torch.arange(n), rot), plain.turn(k, torch.arange(n), rot)
        ref.append((q, k, v))
    state = torch.full((5, taps - 1, width), 0.0, device=DEV)
    tables = scattered_tables([n] * seqs, page, seqs * -(-n // page) + 4, 3)
    k_cache = torch.zeros(seqs * -(-n // page) + 4, nkv, page, d, dtype=dtype, device=DEV)
    v_cache = torch.zeros(k_cache.shape[0], nkv, page, dv, dtype=dtype, device=DEV)
    slots = [4, 0, 2]
    at = [0] * seqs
    tol = lambda r: (1e-5 if dtype == torch.float32 else 2.0 ** -8) * float(r.abs().max())
    for lens in ([11, 1, 2], [2, 2, 2], [1, 1, 1], [1, 9, 1], [1, 1, 1], [14, 16, 3]):
        step = FakeStep(lens, at, slots)
        qkv = torch.cat([raw[i][at[i]:at[i] + m] for i, m in enumerate(lens)]).to(DEV).contiguous()
        pos = step.positions.cpu().double()
        rope = f32(torch.stack([torch.cos(pos[:, None] * freq), torch.sin(pos[:, None] * freq)], dim=-1)) if rd else None
        q_out = torch.empty(sum(lens), nq * d, dtype=dtype, device=DEV)
        ops.conv_rows_norm_cache(qkv, q_out, f32(cw.t()), state, f32(wq), f32(wk), 1e-4, rope, rd, step, tables.to(DEV), k_cache, v_cache,
                                 nq, nkv, d, dv, values_are_keys=keys)
        want = torch.cat([ref[i][0][at[i]:at[i] + m] for i, m in enumerate(lens)])
        assert (q_out.double().cpu().view(-1, nq, d) - want).abs().max() <= tol(want), lens
        at = [a + m for a, m in zip(at, lens)]
    for i in range(seqs):
        assert (rows_of(k_cache, tables[i], page, at[i]) - ref[i][1][:at[i]]).abs().max() <= tol(ref[i][1])
        assert (rows_of(v_cache, tables[i], page, at[i]) - ref[i][2][:at[i]]).abs().max() <= tol(ref[i][2])
        assert torch.equal(state[slots[i]].cpu(), raw[i][at[i] - taps + 1:at[i], :width].float())
    assert float(state[1].abs().max() if taps > 1 else 0) == 0.0 and float(state[3].abs().max() if taps > 1 else 0) == 0.0
    step = FakeStep([1], [3], [-1])                              # a padding row: no slot is touched
    before = state.clone()
    ops.conv_rows_norm_cache(raw[0][:1].to(DEV), torch.empty(1, nq * d, dtype=dtype, device=DEV), f32(cw.t()), state, f32(wq), f32(wk), 1e-4,
                             None, 0, step, torch.full((1, 4), -1, dtype=torch.int32, device=DEV), k_cache, v_cache, nq, nkv, d, dv, values_are_keys=keys)
    assert torch.equal(before, state)


def memory_case(H, d, dv, n, seed, dtype, spread=1.0):
    g = torch.Generator().manual_seed(seed)
    up = lambda c: -(-c // 8) * 8
    cq, ck = 0, up(H * d)
    cv = ck + up(H * d)
    cg = cv + up(H * dv)
    proj = torch.randn(n, cg + up(H * dv) + 8, generator=g).to(dtype)
    gates = torch.randn(n, 2 * H, generator=g) * 4.0 * spread
    bi, bf = torch.linspace(-1.0, 1.0, H) if H > 1 else torch.zeros(1), torch.linspace(0.0, 6.0, H) if H > 1 else torch.full((1,), 3.0)
    return proj, gates, bi, bf, (cq, ck, cv, cg)


def memory_reference(proj, gates, bi, bf, cols, H, d, dv, cap, terms=None):
    n, x = proj.shape[0], proj.double()
    q = x[:, cols[0]:cols[0] + H * d].view(n, H, d) * d ** -0.5
    k, v = x[:, cols[1]:cols[1] + H * d].view(n, H, d), x[:, cols[2]:cols[2] + H * dv].view(n, H, dv)
    z = gates.double()
    i = cap * torch.tanh((z[:, :H] + bi.double()) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((z[:, H:] + bf.double()) / cap))
    return plain.matrix_memory(q, k, v, i, f, terms)


MEMORIES = [(3, 10, 7), (1, 1, 1), (4, 64, 64), (2, 128, 128), (1, 256, 80), (5, 24, 130), (2, 100, 33)]


@pytest.mark.parametrize("H,d,dv", MEMORIES)
@pytest.mark.parametrize("dtype,chunks", [(torch.float32, False), (torch.bfloat16, False), (torch.bfloat16, True)])
@pytest.mark.parametrize("spread", [0.3, 1.5, 8.0])
def test_the_memory_over_portions(H, d, dv, dtype, chunks, spread):
    """Three sequences in two or three portions each (borders inside and at chunks of 64), from the slots of the portions before,
    token by token and 64 tokens at a time; gates from hardly moving to closed and wide open, a cap that bites; slots of others
    stay as they are."""
    from inferloop_b200.csrc import ops
    cap = 7.0
    lens = [150, 65, 40]
    data = [memory_case(H, d, dv, n, 7 * i + d, dtype, spread) for i, n in enumerate(lens)]
    _, _, bi, bf, cols = data[0]
    m = ops.MatrixMemory(H, d, dv, *cols, cap, d ** -0.5, 1e-6, f32(bi), f32(bf))
    refs, bounds = [], []
    for p, z, *_ in data:
        terms = []
        o = memory_reference(p, z, bi, bf, cols, H, d, dv, cap, terms)
        num, nq, den = (torch.stack(x) for x in zip(*terms))
        refs.append(o)
        bounds.append((num + o.abs() * nq[:, :, None]) / den[:, :, None])      # what a rounding of every term amounts to
    state = {"state": torch.zeros(5, H, d, dv, device=DEV), "norm": torch.zeros(5, H, d, device=DEV), "max": torch.zeros(5, H, device=DEV)}
    for t in state.values():
        t[1] = 9.0
    slots, at = [3, 0, 4], [0, 0, 0]
    ws = workspace()
    for portion in ([64, 3, 1], [70, 62, 39], [16]):
        spans = [(i, n) for i, n in enumerate(portion)]
        step = FakeStep([n for _, n in spans], [at[i] for i, _ in spans], [slots[i] for i, _ in spans])
        proj = torch.cat([data[i][0][at[i]:at[i] + n] for i, n in spans]).to(DEV).contiguous()
        gates = f32(torch.cat([data[i][1][at[i]:at[i] + n] for i, n in spans]))
        y = torch.empty(proj.shape[0], H * dv, device=DEV)
        den = ops.mlstm_scan(m, proj, gates, state, y, step, ws, chunks=chunks)
        got = y.double().cpu().view(-1, H, dv)
        if den is not None:
            got = got / den.double().cpu()[:, :, None]
        want = torch.cat([refs[i][at[i]:at[i] + n] for i, n in spans])
        bound = (3e-5 if chunks else 3e-6) * torch.cat([bounds[i][at[i]:at[i] + n] for i, n in spans]) + 1e-12
        assert ((got - want).abs() <= bound).all(), (portion, float(((got - want).abs() / bound).max()))
        for i, n in spans:
            at[i] += n
    assert all(float((t[1] - 9.0).abs().max()) == 0.0 and float(t[2].abs().max()) == 0.0 for t in state.values())


@pytest.mark.parametrize("H,d,dv", MEMORIES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_memory_token_by_token(H, d, dv, dtype):
    """Single tokens from the projections to the gated row in one launch: the gates' dot products, the recurrence, the head's norm
    and the output gate; behind a portion, two sequences, and a padding row without a slot."""
    from inferloop_b200.csrc import ops
    cap, W, n, first = 5.0, 72, 60, 20
    g = torch.Generator().manual_seed(d + dv)
    cases_ = [memory_case(H, d, dv, n, 3 * i + dv, dtype) for i in range(2)]
    _, _, bi, bf, cols = cases_[0]
    x = [torch.randn(n, W, generator=g).to(dtype) for _ in range(2)]
    wg = (torch.randn(2 * H, W, generator=g) * 0.4).to(dtype)
    nw = 1 + 0.2 * torch.randn(H * dv, generator=g)
    m = ops.MatrixMemory(H, d, dv, *cols, cap, d ** -0.5, 1e-6, f32(bi), f32(bf))
    refs, outs = [], []
    for (p, *_), xx in zip(cases_, x):
        gates = xx.double() @ wg.double().T
        o = memory_reference(p, gates, bi, bf, cols, H, d, dv, cap)
        refs.append(plain.rms(o, 1e-5).reshape(n, H * dv) * nw.double() * torch.sigmoid(p.double()[:, cols[3]:cols[3] + H * dv]))
    state = {"state": torch.zeros(3, H, d, dv, device=DEV), "norm": torch.zeros(3, H, d, device=DEV), "max": torch.zeros(3, H, device=DEV)}
    ws = workspace()
    step = FakeStep([first, first], [0, 0], [2, 1])
    proj = torch.cat([p[:first] for p, *_ in cases_]).to(DEV).contiguous()
    gates = f32(torch.cat([xx[:first].double() @ wg.double().T for xx in x]))
    ops.mlstm_scan(m, proj, gates, state, torch.empty(2 * first, H * dv, device=DEV), step, ws, chunks=False)
    wide = torch.zeros(3, H * dv + 5, dtype=dtype, device=DEV)
    for t in range(first, n):
        step = FakeStep([1, 1, 1], [t, t, 0], [2, 1, -1])
        rows = [cases_[0][0][t], cases_[1][0][t], cases_[0][0][0]]
        ops.mlstm_step(m, torch.stack(rows).to(DEV).contiguous(), torch.stack([x[0][t], x[1][t], x[0][0]]).to(DEV).contiguous(), wg.to(DEV), f32(nw),
                       1e-5, state, wide[:, :H * dv], step)
        outs.append(wide[:, :H * dv].double().cpu().clone())
    got = torch.stack(outs)
    for s in range(2):
        want = refs[s][first:]
        # (the head's norm magnifies an output that nearly cancels: one state column is one such number)
        big = want.abs() > 0 if d * dv > 1 else want.abs() >= 0
        tol = (2e-4 if dtype == torch.float32 else 2.0 ** -7) * float(want.abs().max())
        assert ((got[:, s] - want).abs()[big] <= tol).all(), float((got[:, s] - want).abs().max())
        assert (got[:, 2] - refs[0][0]).abs().max() <= tol                    # a row without a slot starts from zero


@pytest.mark.parametrize("rank,tail,rot,heads,K,apart", [(20, 6, 6, 3, 10, True), (96, 32, 32, 4, 64, True), (9, 4, 4, 5, 6, True), (16, 7, 4, 2, 5, True), (32, 9, 6, 2, 8, False),
                                                         (520, 64, 64, 3, 40, True)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_latent_with_a_rotated_part(rank, tail, rot, heads, K, apart, dtype):
    """Latent, rotated key part and the queries' tails in pairs half the rotated part apart (and of neighbours), as a launch of
    its own and inside the input stage of few tokens, which maps the queries too."""
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(rank + tail)
    lens, starts, page = [5, 1, 7], [3, 40, 0], 8
    T = sum(lens)
    step = FakeStep(lens, starts)
    q_cols = heads * (K + tail)
    proj = torch.randn(T, q_cols + rank + tail, generator=g).to(dtype)
    w = 1 + 0.2 * torch.randn(rank, generator=g)
    up = (torch.randn(heads, K, rank, generator=g) / math.sqrt(K)).to(dtype)
    pos = step.positions.cpu()
    freq, _ = plain.frequencies({"base": 30.0, "dims": rot})
    ang = pos.double()[:, None] * freq
    angles = f32(torch.stack([torch.cos(ang), torch.sin(ang)], dim=-1))
    x = proj.double()

    def turned(v):
        if apart:
            return plain.turn(v, pos, {"base": 30.0, "dims": rot})
        c, s = (f(ang).view((T,) + (1,) * (v.dim() - 2) + (rot // 2,)) for f in (torch.cos, torch.sin))
        out = v.clone()
        out[..., 0:rot:2], out[..., 1:rot:2] = v[..., 0:rot:2] * c - v[..., 1:rot:2] * s, v[..., 1:rot:2] * c + v[..., 0:rot:2] * s
        return out
    row = torch.cat([plain.norm(x[:, q_cols:q_cols + rank], w.double(), 1e-4), turned(x[:, q_cols + rank:])], dim=-1)
    q = x[:, :q_cols].view(T, heads, K + tail)
    mapped = torch.cat([torch.einsum("thk,hkr->thr", q[..., :K], up.double()), turned(q[..., K:])], dim=-1)
    tables = scattered_tables([s + n for s, n in zip(starts, lens)], page, 30, 5)
    tol = lambda r: (2e-5 if dtype == torch.float32 else 2.0 ** -7) * float(r.abs().max())
    for fused in (False, True):
        cache = torch.zeros(30, 1, page, rank + tail, dtype=dtype, device=DEV)
        q_out = torch.empty(T, heads * (rank + tail), dtype=dtype, device=DEV)
        pd = proj.to(DEV)
        if fused:
            ops.latent_input(pd, up.to(DEV), q_out, q_cols, rank, f32(w), 1e-4, step, tables.to(DEV), cache, tail, rot, angles, apart)
        else:
            ops.latent_write_rot(pd, q_cols, rank, tail, rot, angles, f32(w), 1e-4, step, tables.to(DEV), cache, pd, q_out, q_col0=K,
                                 q_head_stride=K + tail, heads=heads, half_split=apart)
            ops.head_matmul(pd, up.to(DEV), q_out, x_head_stride=K + tail, out_head_stride=rank + tail)
        assert (q_out.double().cpu().view(T, heads, -1) - mapped).abs().max() <= tol(mapped)
        for i, (n, s) in enumerate(zip(lens, starts)):
            at = sum(lens[:i])
            assert (rows_of(cache, tables[i], page, s + n)[s:, 0] - row[at:at + n]).abs().max() <= tol(row)


@pytest.mark.parametrize("width", [1, 50, 256, 2048, 4100, 5001])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_branches_norms(width, dtype):
    """Two outputs of very different size, each normed by itself: their half sum into a buffer; and normed again, into the stream,
    with the next sublayer's input."""
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    T = 9
    a, b, x = 50 * torch.randn(T, width, generator=g), 0.02 * torch.randn(T, width, generator=g), torch.randn(T, width, generator=g)
    wa, wb, w = (1 + 0.3 * torch.randn(width, generator=g) for _ in range(3))
    z = 0.5 * (plain.norm(a.double(), wa.double(), 1e-5) + plain.norm(b.double(), wb.double(), 1e-5))
    y = f32(x)
    ops.branch_norms_add((f32(a), f32(b)), (f32(wa), f32(wb)), 1e-5, 0.5, y=y)
    assert_close(y, x.double() + z, "float32", "sum")
    xs, out = f32(x), torch.empty(T, width, dtype=dtype, device=DEV)
    ops.branch_norms_add((f32(a), f32(b)), (f32(wa), f32(wb)), 1e-5, 0.5, norm=(f32(w), 3e-5), x=xs, out=out)
    new = x.double() + plain.norm(z, w.double(), 3e-5)
    assert_close(xs, new, "float32", "stream")
    assert_close(out, new, "float32" if dtype == torch.float32 else "bfloat16", "next input")
    xs = f32(x)
    ops.branch_norms_add((f32(a), f32(b)), (f32(wa), f32(wb)), 1e-5, 0.5, norm=(f32(w), 3e-5), x=xs)
    assert_close(xs, new, "float32", "stream alone")


@pytest.mark.parametrize("width,pad", [(9, 3), (64, 8), (300, 4), (2048, 0)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_gate_an_element(width, pad, dtype):
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    o, z = (torch.randn(21, width, generator=g)).to(dtype), (3 * torch.randn(21, width + pad, generator=g)).to(dtype)
    ref = o.double() * torch.sigmoid(z.double()[:, :width])
    wide = torch.full((21, width + 8), 7.0, dtype=dtype, device=DEV)
    ops.gate_rows(o.to(DEV), z.to(DEV), wide[:, :width])
    own = o.to(DEV)
    ops.gate_rows(own, z.to(DEV), own)
    for got in (wide[:, :width], own):
        assert (got.double().cpu() - ref).abs().max() <= (1e-6 if dtype == torch.float32 else 2.0 ** -8) * float(ref.abs().max())
    assert (wide[:, width:] == 7.0).all()


@pytest.mark.parametrize("M,K,I", [(1, 64, 64), (8, 256, 128), (33, 72, 192), (300, 256, 512), (2048, 512, 1024)])
def test_gelu_inside_the_product_and_alone(M, K, I):
    """The gated unit with gelu's tanh form in the tensor-core product's epilogue (every form: few tokens, clusters, many tokens,
    pairs of CTAs) and as a kernel of its own, gates from far below zero to far above."""
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(M + I)
    a = torch.randn(M, K, generator=g).to(torch.bfloat16)
    gate, up = (3 * torch.randn(I, K, generator=g) / math.sqrt(K)).to(torch.bfloat16), (torch.randn(I, K, generator=g) / math.sqrt(K)).to(torch.bfloat16)
    w = torch.stack([gate.view(I // 64, 64, K), up.view(I // 64, 64, K)], dim=1).reshape(2 * I, K).contiguous()
    zg, zu = a.double() @ gate.double().T, a.double() @ up.double().T
    ref = plain.gelu_tanh(zg) * zu
    for pairs in (0, 1, 2):
        ops.gemm_pairs(pairs)
        try:
            out = torch.full((M, I), 9.0, dtype=torch.bfloat16, device=DEV)
            ops.gemm_tc(a.to(DEV), w.to(DEV), out, swiglu=True, gate="gelu_tanh")
            assert ((out.double().cpu() - ref).abs() <= 2.0 ** -7 * ref.abs() + 2e-4 * (1 + zu.abs())).all()
        finally:
            ops.gemm_pairs(1)
    for dtype in (torch.float32, torch.bfloat16):
        x = torch.cat([zg, zu], dim=1).to(dtype)
        out = torch.empty(M, I, dtype=dtype, device=DEV)
        ops.silu_mul(x.to(DEV).contiguous(), out, "gelu_tanh")
        want = plain.gelu_tanh(x.double()[:, :I]) * x.double()[:, I:]
        assert ((out.double().cpu() - want).abs() <= (2e-6 if dtype == torch.float32 else 2.0 ** -8) * want.abs() + 1e-5).all()


@pytest.mark.parametrize("experts,top,groups,keep", [(6, 2, 3, 2), (12, 3, 2, 1), (8, 1, 4, 1), (20, 4, 5, 2), (64, 6, 8, 3), (96, 8, 4, 2), (512, 8, 16, 4), (5, 3, 1, 1), (4, 2, 4, 2)])
@pytest.mark.parametrize("best_two", [True, False])
def test_groups_ranked_by_their_two_best(experts, top, groups, keep, best_two):
    """Sigmoid scores with a correction that pushes choice scores below zero; among the rows some whose best group by its best
    member and by its two best together differ, and some with equal members (the second best may equal the best)."""
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(experts + top)
    T, per = 97, experts // groups
    z = 2 * torch.randn(T, experts, generator=g)
    corr = torch.linspace(-0.4, 0.2, experts) - 0.5
    if groups > 1 and per > 1:
        z[:20] = -3.0
        corr = torch.zeros(experts) - 0.5
        for t in range(20):
            a, b = t % groups, (t + 1) % groups
            z[t, a * per] = 2.0                                  # the single best
            z[t, b * per:b * per + 2] = 1.2                      # two good ones of one value
    choice, weight = torch.empty(T * top, dtype=torch.int32, device=DEV), torch.empty(T * top, device=DEV)
    ops.moe_route(f32(z), experts, top, False, False, choice, weight, correction=f32(corr), groups=groups, keep=keep, group_best_two=best_two)
    scores = torch.sigmoid(z.double())
    c = scores + corr.double()
    if not best_two:
        rank = c.view(T, groups, per).max(-1).values
    else:
        rank = plain.group_scores(c, groups)
    best = torch.argsort(rank, dim=-1, descending=True, stable=True)[:, :keep]
    allowed = torch.zeros(T, groups, dtype=torch.bool).scatter_(1, best, True).repeat_interleave(per, dim=1)
    order = torch.argsort(c.masked_fill(~allowed, float("-inf")), dim=-1, descending=True, stable=True)[:, :top]
    if best_two and groups > 1:
        assert torch.equal(order, plain.route(scores, corr.double(), top, {"count": groups, "keep": keep})[0])
    got = choice.cpu().view(T, top).long()
    assert torch.equal(torch.sort(got, -1).values, torch.sort(order, -1).values)
    assert (weight.double().cpu().view(T, top) - scores.gather(1, got)).abs().max() < 1e-6


@pytest.mark.parametrize("heads,dv", [(1, 9), (3, 10), (8, 64), (2, 128), (5, 300)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_norm_of_each_head_divided_by_a_number_first(heads, dv, dtype):
    """eps sits inside the root, so dividing a head's output first is not the same as leaving it to the norm."""
    from inferloop_b200.csrc import ops
    g = torch.Generator().manual_seed(heads * dv)
    T, width = 11, heads * dv
    y, den = torch.randn(T, width, generator=g), torch.logspace(-2, 4, T * heads).view(T, heads)
    z, w = torch.randn(T, width + 4, generator=g).to(dtype), 1 + 0.2 * torch.randn(width, generator=g)
    out = torch.empty(T, width, dtype=dtype, device=DEV)
    ops.rms_gate(f32(y), z.to(DEV), f32(w), 1e-5, out, groups=heads, divisor=f32(den))
    o = y.double().view(T, heads, dv) / den.double()[:, :, None]
    ref = plain.rms(o, 1e-5).reshape(T, width) * w.double() * torch.sigmoid(z.double()[:, :width])
    assert (out.double().cpu() - ref).abs().max() <= (1e-5 if dtype == torch.float32 else 2.0 ** -8) * float(ref.abs().max())
