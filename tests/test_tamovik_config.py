"""The Tamovik configuration, its mapping to a model description, what its layers ask of the cache manager, and its plain
statement on cases worked by hand (no GPU)."""
import copy
import json
import math

import pytest
import torch

import plain_tamovik as plain
import tamovik_cases as cases
from inferloop_b200.cache import CacheManager
from inferloop_b200.config import ConfigError, UnsupportedConfig, read_model_config
from inferloop_b200.config.tamovik import TamovikConfig
from inferloop_b200.models.decoder import DecoderModel, declare_weights
from inferloop_b200.parts.base import BuildContext, PagedKVNeed, Workspace


def spec_of(config):
    return read_model_config(json.dumps(config))[2]


def test_the_mapping():
    spec = spec_of(cases.CONFIG_K)
    assert spec.architecture == "Tamovik" and spec.head_name == "head" and spec.embedding.kind == "hashed_pairs"
    assert (spec.embedding["buckets"], spec.embedding["mul_prev"], spec.embedding["mul_cur"]) == (101, 13, 5)
    assert spec.final_norm.kind == "rms" and spec.logits_post is None and spec.final_norm["eps"] == 1e-5
    assert [l.block.kind for l in spec.layers] == ["output_norm"] * 4
    assert [l.mixer.kind for l in spec.layers] == ["latent_attention", "parallel", "parallel", "latent_attention"]
    assert [l.feed_forward.kind for l in spec.layers] == ["swiglu", "routed_experts", "none", "routed_experts"]
    m = spec.layers[0].mixer
    assert m["position"].kind == "rope_neox" and m["position"]["ramp"] == (4.0, 60.0, 8.0, 1.0) and m["rot_dim"] == 6 and m["latent"] == 20
    assert spec.layers[3].mixer["position"]["ramp"] is None
    (lp, left), (rp, right) = spec.layers[1].mixer["branches"]
    assert (lp, rp) == ("left.", "right.") and left.kind == "gqa_attention" and right.kind == "mlstm"
    assert left["chunk"] == 13 and left["conv"] == 5 and left["values"] == "keys" and left["output_gate"] == "element" and left["qk_norm"] == "rows"
    assert left["position"].kind == "none" and right["gate_cap"] == 4.0 and right["den_eps"] == 1e-6
    assert spec.layers[1].mixer["out_norms"] == ("left.out", "right.out") and spec.layers[1].mixer["out_mult"] == 0.5
    assert spec.layers[0].feed_forward["activation"] == "gelu_tanh"
    f = spec.layers[1].feed_forward
    assert f["groups"] == (3, 2) and f["group_rank"] == "best_two" and f["score"] == "sigmoid" and not f["renormalize"] and f["correction"]
    assert f["activation"]["limit"] == 0.8 and f["activation"]["sharpness"] == 1.702 and f["activation"]["up_offset"] == 1.0
    assert spec.layers[3].feed_forward["groups"] is None
    n = spec_of(cases.CONFIG_N)
    assert n.embedding is None and n.layers[0].mixer["branches"][0][1]["chunk"] is None


def test_the_declared_tensors_and_their_shapes():
    decl = {d.name: tuple(d.shape) for d in declare_weights(spec_of(cases.CONFIG_K))}
    assert decl["embed"] == decl["head"] == (203, 72) and decl["bigram"] == (102, 72) and decl["final.norm"] == (72,)
    assert decl["l0.mix.q"] == (48, 72) and decl["l0.mix.dkv"] == (26, 72) and decl["l0.mix.dkv.norm"] == (20,)
    assert decl["l0.mix.uk"] == (30, 20) and decl["l0.mix.uv"] == (21, 20) and decl["l0.mix.o"] == (72, 21)
    assert decl["l1.mix.left.q"] == (72, 72) and decl["l1.mix.left.k"] == (24, 72) and "l1.mix.left.v" not in decl
    assert decl["l1.mix.left.q.conv"] == (72, 5) and decl["l1.mix.left.k.conv"] == (24, 5)
    assert decl["l1.mix.left.q.norm"] == (72,) and decl["l1.mix.left.k.norm"] == (24,) and decl["l1.mix.left.g"] == (72, 72)
    assert decl["l1.mix.right.q"] == decl["l1.mix.right.k"] == (30, 72) and decl["l1.mix.right.v"] == decl["l1.mix.right.g"] == (21, 72)
    assert decl["l1.mix.right.i"] == decl["l1.mix.right.f"] == (3, 72) and decl["l1.mix.right.i.b"] == (3,) and decl["l1.mix.right.norm"] == (21,)
    assert decl["l1.mix.left.out"] == decl["l1.mix.right.out"] == (72,)
    assert decl["l0.mlp.gate"] == (52, 72) and decl["l1.mlp.router"] == (6, 72) and decl["l1.mlp.correction"] == (6,) and decl["l1.mlp.e5.down"] == (72, 20)
    optional = {d.name for d in declare_weights(spec_of(cases.CONFIG_K)) if d.optional}
    assert optional == {"l2.norm2"}


@pytest.mark.parametrize("change,error", [
    (lambda c: c["layers"][0].update(type="attention"), UnsupportedConfig),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), ConfigError),
    (lambda c: c["layers"][0]["mixer"].update(kv_rank=700), UnsupportedConfig),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=8), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=0), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), ConfigError),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), ConfigError),
    (lambda c: c["layers"][1]["mixer"].pop("right"), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["left"].update(vdim=10), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["left"].update(conv=0), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["left"].update(conv=17), UnsupportedConfig),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["right"].update(gate_cap=0), ConfigError),
    (lambda c: c["layers"][1]["mixer"]["right"].update(dim=257), UnsupportedConfig),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), ConfigError),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), ConfigError),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), ConfigError),
    (lambda c: c["layers"][1]["mlp"]["expert"].update(limit=0), ConfigError),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), UnsupportedConfig),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), ConfigError),
    (lambda c: c["embedding"]["bigram"].pop("mul_cur"), ConfigError),
    (lambda c: c["norm"].update(eps=0), ConfigError),
    (lambda c: c.pop("width"), ConfigError),
    (lambda c: c.update(layers=[]), ConfigError),
])
def test_refusals(change, error):
    config = copy.deepcopy(cases.CONFIG_K)
    change(config)
    with pytest.raises(error):
        read_model_config(json.dumps(config))


def test_what_is_absent_from_the_file_is_absent_from_the_model():
    config = copy.deepcopy(cases.CONFIG_K)
    config.pop("embedding")
    config["layers"][0]["mixer"]["rot"].pop("scaling")
    config["layers"][1]["mixer"]["left"].pop("mask")
    config["layers"][1]["mlp"]["router"].pop("groups")
    cfg = TamovikConfig.from_dict(config)
    assert cfg.pairs is None and cfg.layers[0].mixer.rot.scaling is None and cfg.layers[1].mixer.left.chunk is None
    assert cfg.layers[1].mlp.groups == 1 and cfg.layers[2].mlp is None
    assert spec_of(config).embedding is None


def test_what_the_layers_ask_of_the_cache_manager():
    """A latent layer: one row of latent and rotated part a token; a parallel layer: keys and values no longer than a chunk back,
    the convolution's last inputs, and state, normaliser and maximum under their branch's number."""
    spec = spec_of(cases.CONFIG_K)
    model = DecoderModel(spec, BuildContext(torch.float32, None, Workspace(None)))
    needs = model.cache_needs()
    assert needs[0].paged == PagedKVNeed(1, 26, None, 0) and needs[0].slots == ()
    assert needs[1].paged == PagedKVNeed(2, 12, 13) and needs[2].paged == PagedKVNeed(3, 6, 30)
    assert [(s.name, s.shape) for s in needs[1].slots] == [("0.conv", (4, 96)), ("1.state", (3, 10, 7)), ("1.norm", (3, 10)), ("1.max", (3,))]
    assert [s.name for s in model.model_slot_needs()] == ["previous_token"]
    m = CacheManager(needs, page_size=4, num_pages=20, max_requests=2, run_order=spec.run_order)
    assert len(m.groups) == 4
    m.begin("a"); m.ensure("a", 27); m.commit("a", 27)
    m.ensure("a", 28)                                    # position 27 is in the chunk 26 .. 38
    assert m.block_table(1, "a")[6:] and min(m.block_table(1, "a")[6:]) >= 0 and m.block_table(1, "a")[0] == -1
    m.commit("a", 28); m.release("a")
    m.check()
    n = DecoderModel(spec_of(cases.CONFIG_N), BuildContext(torch.float32, None, Workspace(None)))
    assert n.cache_needs()[0].paged.window is None and n.model_slot_needs() == ()


def test_the_plain_statement_on_cases_worked_by_hand():
    d = lambda *v: torch.tensor(v, dtype=torch.float64)
    # groups by their two best together: 0.5 + 0.4 beats 0.8 + 0.0 although the single best is in the other group
    scores = d([0.8, 0.0, 0.5, 0.4])
    chosen, weights = plain.route(scores, d(0, 0, 0, 0), 2, {"count": 2, "keep": 1})
    assert chosen.tolist() == [[2, 3]] and weights.tolist() == [[0.5, 0.4]]
    chosen, weights = plain.route(scores, d(-2.0, -2.0, -2.0, -2.0), 2, {"count": 2, "keep": 1})        # every ranking score negative
    assert chosen.tolist() == [[2, 3]] and weights.tolist() == [[0.5, 0.4]]
    chosen, weights = plain.route(scores, d(0, 0.9, 0, 0), 1, {"count": 2, "keep": 1})
    assert chosen.tolist() == [[1]] and weights.tolist() == [[0.0]]                                     # ranked by s + c, weighted by s
    assert plain.route(scores, d(0, 0, 0, 0), 3, None)[0].tolist() == [[0, 2, 3]]
    # chunks are counted from position 0
    seen = plain.same_chunk(7, 3)
    assert [seen[i].nonzero().flatten().tolist() for i in (2, 3, 5, 6)] == [[0, 1, 2], [3], [3, 4, 5], [6]]
    # a convolution of two taps: w0 u_{t-1} + w1 u_t
    y = plain.short_conv(d([1.0], [10.0], [100.0]), d([2.0, 3.0]))
    assert y.flatten().tolist() == [3.0, 32.0, 320.0]
    # the memory's maximum starts at zero: one weak token of weight exp(i) leaves m = f if i < f < 0
    one = lambda v: d(v).view(1, 1, 1)
    i, f = d([-5.0]).view(1, 1), d([-1.0]).view(1, 1)
    o = plain.matrix_memory(one(2.0), one(3.0), one(7.0), i, f)
    n = math.exp(-5.0 + 1.0) * 3.0
    assert abs(float(o) - n * 7.0 * 2.0 / (max(2.0 * n, math.e) + 1e-6)) < 1e-12
    # the first token has no pair; pairs are (previous, token)
    w = {"embed": torch.zeros(9, 1, dtype=torch.float64), "bigram": torch.arange(6.0, dtype=torch.float64)[:, None]}
    e = plain.embedding(w, {"embedding": {"bigram": {"buckets": 5, "mul_prev": 3, "mul_cur": 2}}}, [4, 1, 8])
    assert e.flatten().tolist() == [5.0, float((12 + 2) % 5), float((3 + 16) % 5)]
    # a ramp over the pairs: the first is kept, the last divided
    f, stretch = plain.frequencies({"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 256, "fast": 16.0, "slow": 1.0}})
    assert f[0] == 1.0 and abs(float(f[-1]) * 8.0 - 10000.0 ** (-62 / 64)) < 1e-12 and abs(stretch - (1 + 0.1 * math.log(8.0))) < 1e-15


MISTAKES = {
    "a chunk one position longer": ("same_chunk", lambda f: lambda n, size: f(n, size + 1)),
    "a chunk one position shorter": ("same_chunk", lambda f: lambda n, size: f(n, max(size - 1, 1))),
    "a window instead of a chunk": ("same_chunk", lambda f: lambda n, size: plain.causal(n) & (torch.arange(n)[:, None] - torch.arange(n)[None, :] < size)),
    "taps in the other order": ("short_conv", lambda f: lambda u, w: f(u, w.flip(1))),
    "a convolution that forgets the token before": ("short_conv", lambda f: lambda u, w: u * w[:, -1]),
    "cos and sin not stretched": ("frequencies", lambda f: lambda rot: (f(rot)[0], 1.0)),
    "frequencies not blended": ("frequencies", lambda f: lambda rot: (f({k: v for k, v in rot.items() if k != "scaling"})[0], f(rot)[1])),
    "positions one off for the keys' part alone": ("turn", lambda f: lambda x, p, rot: f(x, p + (1 if x.dim() == 2 else 0), rot)),
    "groups by their best member": ("group_scores", lambda f: lambda c, n: c.view(c.shape[0], n, -1).max(-1).values),
    "weights that carry the correction": ("route", lambda f: lambda s, c, top, g: (f(s, c, top, g)[0], (s + c).gather(1, f(s, c, top, g)[0]))),
    "a memory that starts anew every 32 tokens": ("matrix_memory", lambda f: lambda q, k, v, i, g, terms=None: torch.cat(
        [f(*(x[a:a + 32] for x in (q, k, v, i, g))) for a in range(0, q.shape[0], 32)])),
    "a forget gate without its logarithm's bend": ("mlstm_gates", lambda f: lambda w, p, m, h: (f(w, p, m, h)[0], f(w, p, m, h)[1] * 0.9)),
    "gates without a cap": ("mlstm_gates", lambda f: lambda w, p, m, h: f(w, p, dict(m, gate_cap=1e3), h)),
    "branches added without their norms": ("norm", lambda f: lambda x, w, eps: f(x, w, eps) if x.shape[-1] != 72 or w is not LEFT[0] else x),
}
LEFT = [None]
SMALL = ("cos and sin not stretched", "a forget gate without its logarithm's bend")


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_the_cases_show_a_planted_mistake(mistake, monkeypatch, tmp_path_factory):
    """A mistake in the statement itself moves some position's logits far beyond what a comparison allows: the weights of case K
    do not hide it.  (Two of them are small by nature: those have to stand out of what a 32-bit comparison allows.)"""
    model = cases.plain_model(str(tmp_path_factory.mktemp("tamovik")), "K", torch.float32)
    LEFT[0] = model.w["l1.mix.left.out"]
    tokens = [(7 * i * i + 3 * i) % 203 for i in range(80)]
    ref = model.forward(tokens)
    name, wrong = MISTAKES[mistake]
    monkeypatch.setattr(plain, name, wrong(getattr(plain, name)))
    err = (model.forward(tokens) - ref).pow(2).mean(-1).sqrt() / float(ref.abs().max())
    most, many = (1e-3, 1e-4) if mistake in SMALL else (0.06, 0.01)
    assert float(err.max()) > most and int((err > many).sum()) > 8, (float(err.max()), int((err > many).sum()))
