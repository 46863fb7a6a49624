"""The Sapanex configuration, its mapping to a model description, what its layers ask of the cache manager, tensors whose
size the file decides, and the plain statement on cases worked by hand (no GPU)."""
import copy
import json
import math
import random

import pytest
import torch

import plain_sapanex as plain
import sapanex_cases as cases
from fake_runner import FakeRunner
from helpers import random_tokens
from inferloop_b200.cache import CacheManager
from inferloop_b200.config import ConfigError, UnsupportedConfig, read_model_config
from inferloop_b200.config.sapanex import SapanexConfig
from inferloop_b200.config.spec import PartSpec
from inferloop_b200.engine.engine import Engine
from inferloop_b200.engine.scheduler import CapacityError
from inferloop_b200.models.decoder import DecoderModel, declare_weights
from inferloop_b200.parts import registry
from inferloop_b200.parts.base import BuildContext, CacheNeeds, PagedKVNeed, Workspace
from inferloop_b200.weights.decl import FreeDim, WeightDecl, shapes_agree
from inferloop_b200.weights.loader import WeightError, load_weights


def spec_of(config):
    return read_model_config(json.dumps(config))[2]


def test_the_mapping():
    spec = spec_of(cases.CONFIG_K)
    assert spec.architecture == "Sapanex" and spec.head_name is None and spec.embedding_scale == 2.5 and spec.final_norm.kind == "rms"
    assert [l.block.kind for l in spec.layers] == ["sum_norm"] * 4 and spec.layers[0].block["alpha"] == 1.7
    assert [l.mixer.kind for l in spec.layers] == ["general_delta", "gqa_attention", "general_delta", "gqa_attention"]
    assert [l.feed_forward.kind for l in spec.layers] == ["two_matrix", "two_matrix", "none", "none"]
    a = spec.layers[1].mixer
    assert a["qk_norm"] == "rows" and a["window"] == 7 and a["pool"] == 3 and a["scale"] == 0.5 and a["v_head_dim"] == 10
    assert a["position"]["ramp"] == (4.0, 60.0, 8.0, 1.0) and a["position"]["rotary_dim"] == 8
    assert a["value_position"]["rotary_dim"] == 10 and a["value_position"].get("ramp") is None and a["value_position"]["theta"] == 30.0
    assert spec.layers[0].mixer["log_decay"] == math.exp(-0.5) and spec.layers[0].mixer["unit_eps"] == 1e-6
    assert spec.layers[0].feed_forward["activation"] == "relu2"
    o = spec_of(cases.CONFIG_O)
    assert o.layers[0].mixer["window"] is None and o.layers[0].mixer["pool"] is None and o.layers[1].mixer["position"]["ramp"] is None
    assert o.layers[2].mixer["position"].kind == "none" and o.layers[2].mixer["value_position"].kind == "none"
    config = copy.deepcopy(cases.CONFIG_K)
    config.pop("embedding")
    assert SapanexConfig.from_dict(config).embedding_scale == 1.0


def test_the_declared_tensors_and_their_shapes():
    decls = declare_weights(spec_of(cases.CONFIG_K))
    decl = {d.name: tuple(d.shape) for d in decls}
    assert decl["embed"] == (203, 72) and decl["final.norm"] == (72,) and "head" not in decl
    assert decl["l0.mix.r"] == decl["l0.mix.k"] == decl["l0.mix.v"] == decl["l0.mix.g"] == decl["l0.mix.a"] == (30, 72)
    assert decl["l0.mix.a.b"] == decl["l0.mix.w0"] == decl["l0.mix.norm"] == (30,) and decl["l0.mix.o"] == (72, 30)
    assert decl["l0.mix.w1"][1] == 72 and decl["l0.mix.w2"][0] == 30 and isinstance(decl["l0.mix.w1"][0], FreeDim)
    assert decl["l1.mix.q"] == (60, 72) and decl["l1.mix.k"] == (12, 72) and decl["l1.mix.v"] == (10, 72) and decl["l1.mix.o"] == (72, 50)
    assert decl["l1.mix.q.norm"] == (60,) and decl["l1.mix.k.norm"] == (12,)
    assert decl["l0.mlp.up"] == (40, 72) and decl["l0.mlp.down"] == (72, 40) and "l2.mlp.up" not in decl
    optional = {d.name for d in decls if d.optional}
    assert optional == {"l2.norm2", "l3.norm2"}                    # a layer without feed-forward: its second norm may be stored


@pytest.mark.parametrize("change,error", [
    (lambda c: c["layers"][0].update(type="delta"), UnsupportedConfig),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=2), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=14), ConfigError),
    (lambda c: c["layers"][1]["mixer"].update(vdim=9), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["mask"].pop("pool"), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), ConfigError),
    (lambda c: c["layers"][1]["mixer"].update(dim=600), UnsupportedConfig),
    (lambda c: c["layers"][0]["mixer"].update(dim=300), UnsupportedConfig),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), UnsupportedConfig),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), ConfigError),
    (lambda c: c["norm"].update(eps=0), ConfigError),
    (lambda c: c.pop("postln_alpha"), ConfigError),
    (lambda c: c.pop("width"), ConfigError),
    (lambda c: c.update(layers=[]), ConfigError),
])
def test_refusals(change, error):
    config = copy.deepcopy(cases.CONFIG_K)
    change(config)
    with pytest.raises(error):
        read_model_config(json.dumps(config))


def test_a_dimension_that_the_stored_tensor_decides(tmp_path):
    """The inner size of the decays' map is whatever the file's two matrices agree on, and an error where they do not."""
    folder = cases.folder(str(tmp_path), "K", torch.float32)
    decls = declare_weights(spec_of(cases.CONFIG_K))
    tensors, _ = load_weights(folder, decls, ("",), "embed", torch.float32, "cpu")
    assert tensors["l0.mix.w1"].shape == (5, 72) and tensors["l0.mix.w2"].shape == (30, 5)
    found = {}
    assert shapes_agree((FreeDim(3, "x"), 7), (9, 7), found) and found == {"x": 9}
    assert not shapes_agree((2, FreeDim(3, "x")), (2, 8), found) and shapes_agree((2, FreeDim(3, "x")), (2, 9), found)
    assert not shapes_agree((FreeDim(3, "y"), 7), (9, 6), {}) and not shapes_agree((FreeDim(3, "y"),), (9, 6), {})
    other = [WeightDecl(d.name, (30, FreeDim(4, "l0.mix.w1")) if d.name == "l1.mix.q" else d.shape, d.role, d.init, d.root, d.optional) for d in decls]
    with pytest.raises(WeightError, match="l1.mix.q"):
        load_weights(folder, other, ("",), "embed", torch.float32, "cpu")


def test_what_the_layers_ask_of_the_cache_manager():
    spec = spec_of(cases.CONFIG_K)
    model = DecoderModel(spec, BuildContext(torch.float32, None, Workspace(None)))
    needs = model.cache_needs()
    assert needs[0].paged is None and [(s.name, s.shape) for s in needs[0].slots] == [("state", (3, 10, 10))]
    assert needs[1].paged == PagedKVNeed(1, 12, 7, 10) and needs[1].pooled == PagedKVNeed(1, 12, None, 10, 3)
    assert needs[3].paged == PagedKVNeed(4, 6, 9, 14) and needs[3].pooled == PagedKVNeed(4, 6, None, 14, 9)     # a block outlives the window
    m = CacheManager(needs, page_size=4, num_pages=12, max_requests=2, run_order=spec.run_order)
    assert [g.need.stride for g in m.groups] == [1, 3, 1, 9]
    assert [g.pool.num_pages for g in m.groups] == [12, 4 + 2, 12, 2 + 2]
    assert CacheManager.group_needs(needs, spec.run_order) == [(g.need, g.layers) for g in m.groups]


@pytest.mark.parametrize("seed", range(6))
def test_pages_whose_rows_stand_for_several_tokens(seed):
    """A random life of several requests: a pooled group holds a page per page_size * stride tokens once they are there, never
    more and never fewer; a windowed group beside it lets pages go only when the window and the unfinished block have passed
    them; what ends gives everything back."""
    rng = random.Random(seed)
    stride, window, page = rng.choice([1, 2, 5, 12]), rng.choice([1, 4, 9, 30]), rng.choice([2, 4, 8])
    need = CacheNeeds(paged=PagedKVNeed(1, 8, max(window, stride)), pooled=PagedKVNeed(1, 8, None, None, stride))
    m = CacheManager([need, need], page_size=page, num_pages=200, max_requests=3)
    assert len(m.groups) == 2 and m.groups[0].layers == m.groups[1].layers == [0, 1]
    length = {}
    for _ in range(150):
        if len(length) < 3 and rng.random() < 0.3:
            r = f"r{rng.random()}"
            m.begin(r)
            length[r] = 0
        elif length and rng.random() < 0.1:
            r = rng.choice(list(length))
            m.release(r)
            del length[r]
        elif length:
            r = rng.choice(list(length))
            old, new = length[r], length[r] + rng.randrange(1, 25)
            if sum(-(-(n + 60) // page) for n in length.values()) > 190:
                m.release(r)
                del length[r]
                continue
            expected = m.pages_needed(r, new)
            free = m.free_pages()
            m.ensure(r, new)
            assert {g: free[g] - m.free_pages()[g] for g in free} == expected
            tokens, rows = m.block_table(0, r), m.block_table(1, r)
            assert len(tokens) == -(-new // page) and len(rows) == -(-(new // stride) // page) and min(rows, default=0) >= 0
            # every key that a token of this step, or the mean of a block it completes, reads
            first = min(max(0, old - window + 1), old // stride * stride)
            assert all(p >= 0 for p in tokens[first // page:])
            m.commit(r, new)
            length[r] = new
        m.check()
    for r in list(length):
        m.release(r)
    m.check()
    assert all(n == g.pool.num_pages for g, n in zip(m.groups, m.free_pages().values()))


def test_the_scheduler_counts_rows_of_pooled_groups():
    """A request whose blocks the pooled pages cannot hold is refused, one that just fits is not; under page pressure on the
    pooled group alone requests are preempted and every one still draws the tokens it draws alone."""
    need = [CacheNeeds(paged=PagedKVNeed(1, 8, 6), pooled=PagedKVNeed(1, 8, None, None, 4))]

    def engine(pages):
        return Engine(None, runner=FakeRunner(page_size=2, num_pages=pages, max_requests=4, needs=need), max_num_seqs=4, prefill_chunk_tokens=8,
                      max_num_batched_tokens=12)

    e = engine([60, 3])
    with pytest.raises(CapacityError):
        e.submit(list(range(25)), None, 7, request_id="big")                # 32 tokens: 8 rows, 4 pages
    e.submit(list(range(20)), None, 7, request_id="fits")                    # 27 tokens: 6 rows, 3 pages
    while not e.is_idle():
        e.step()
    assert len(e.result("fits").generated) == 7
    prompts = [random_tokens(n, 50, 300 + n) for n in (17, 9, 23, 14, 5)]
    alone = []
    for i, p in enumerate(prompts):
        one = engine([60, 40])
        one.submit(p, None, 12, request_id=i)
        while not one.is_idle():
            one.step()
        alone.append(one.result(i).generated)
    e = engine([60, 9])
    for i, p in enumerate(prompts):
        e.submit(p, None, 12, request_id=i)
    while not e.is_idle():
        e.step()
    assert [e.result(i).generated for i in range(5)] == alone
    assert e.scheduler.stats["preemptions"] > 0
    assert e.runner.cache.free_pages() == {0: 60, 1: 9}


def test_frequencies_along_a_ramp():
    """The three kinds of pair (kept, blended, divided) against the plain statement, and what cos and sin are stretched by."""
    ctx = BuildContext(dtype=torch.float32, device=torch.device("cpu"), workspace=Workspace(torch.device("cpu")))
    for base, dims, ramp in ((30.0, 8, (4.0, 60.0, 8.0, 1.0)), (10000.0, 64, (8.0, 256.0, 16.0, 1.0)), (1e6, 48, (40.0, 4096.0, 32.0, 1.0)),
                             (3000.0, 128, (2.0, 64.0, 4.0, 0.5)), (7.0, 2, (2.0, 16.0, 4.0, 1.0)), (300.0, 12, None)):
        part = registry.build("position", PartSpec.make("rope_neox", theta=base, rotary_dim=dims, ramp=ramp), ctx)
        want, stretch = plain.frequencies(base, dims, None if ramp is None else dict(zip(("factor", "original", "fast", "slow"), ramp)))
        assert torch.allclose(part.inv_freq(), want, rtol=1e-14, atol=0) and abs(part.stretch - stretch) < 1e-15
        bare, one = plain.frequencies(base, dims)
        assert one == 1.0
        if ramp is not None and dims > 8:
            ratio = want / bare
            assert (ratio > 0.999).any() and (ratio < 1.001 / ramp[0]).any() and ((ratio > 1.01 / ramp[0]) & (ratio < 0.99)).any()
    with pytest.raises(ValueError):
        registry.build("position", PartSpec.make("rope_neox", theta=10.0, rotary_dim=4, ramp=(2.0, 8.0, 1.0, 1.0), scaling=(2.0, 1.0, 4.0, 8.0)), ctx)


def test_the_plain_statement_on_cases_worked_by_hand():
    tok, blk = plain.visible(12, 4, 3)
    assert tok[7].nonzero().flatten().tolist() == [4, 5, 6, 7]
    assert blk[5].tolist() == [False] * 4 and blk[6].tolist() == [True, False, False, False]        # block 0 ends at 2 = 6 - 4
    assert blk[9].tolist() == [True, True, False, False] and blk[8].tolist() == [True, False, False, False]     # 3 and 4 left, their block is not seen
    k = torch.arange(7.0, dtype=torch.float64)[:, None, None]
    assert plain.block_means(k, 3).flatten().tolist() == [1.0, 4.0]
    # one channel: S = w S - a u (u S) + k v with u = k / sqrt(k^2 + 1e-6)
    one = lambda *v: torch.tensor(v, dtype=torch.float64)[:, None, None]
    o, S = plain.delta_rule(one(0.5, 0.5), one(1.0, 0.25), one(2.0, -1.0), one(3.0, 1.0), one(1.0, 2.0))
    assert abs(float(o[0]) - 6.0) < 1e-5 and abs(float(S) - (0.5 * 6 - 0.25 * 6 - 1.0)) < 1e-5 and abs(float(o[1]) - 2 * float(S)) < 1e-12
    # a value turned by its own position and the output turned back by the query's: a rotation by the difference
    f, _ = plain.frequencies(10.0, 2)
    v = torch.tensor([[[1.0, 0.0]]], dtype=torch.float64)
    back = plain.turn(plain.turn(v, torch.tensor([5]), f), torch.tensor([8]), f, sign=-1.0)
    assert torch.allclose(back, torch.tensor([[[math.cos(-3.0), math.sin(-3.0)]]], dtype=torch.float64))
