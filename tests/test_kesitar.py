"""The Kesitar design in the engine against the plain implementation (tests/plain_kesitar.py).

Every test makes its own small configuration and weights (tests/kesitar_util.py).  The CPU tests put the plain
PyTorch stand-ins of the kernels (tests/kernel_refs.py) under the engine, so they test what is host logic:
configuration, registry, tensor names, caches of tokens and of blocks, values handed from layer to layer, batching.
The GPU tests run the same traces on the kernels, in float32 and bfloat16: every mechanism alone, whole prompts, prompts
followed by token-by-token decoding (from CUDA graphs), portions down to one and two tokens, mixed batches of unequal
requests with pages and state slots that are used again, peaky attention at every edge of windows, blocks and pages,
the sink at the first tokens, a far block that decides, a state that remembers, and greedy generation through
``Engine.generate``.
"""
import copy
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import kesitar_util as U
import plain_kesitar as P
import replay_util as ru

DEV = "cuda:0"
# float32: the engine against 64-bit arithmetic, both from the same bfloat16-representable weights, relative to a
# row's largest logit.  bfloat16: products and activations are rounded to 8 bits of mantissa between kernels, and
# the tests' peaky attention (so that a lost key shows) multiplies the rounding of q and k by the scores' spread.
TOL = {torch.float32: dict(rtol=5e-5, atol=1e-6), torch.bfloat16: dict(rtol=8e-2, atol=4e-3)}


def make_runner(tmp_path, cfg, weights, dtype, device, **kw):
    from zinfer_b200.engine import ModelRunner

    d = U.write_model(str(tmp_path / f"m{abs(hash(json.dumps(cfg, sort_keys=True))) % 10**8}"), cfg, weights)
    kw.setdefault("page_size", 8)
    kw.setdefault("max_requests", 4)
    return ModelRunner.from_model_dir(d, dtype=dtype, device=device, **kw)


# ============================================================================ CPU
def test_config_is_read_and_registered():
    from zinfer_b200.config import ConfigError, KesitarConfig, family_for, kesitar_model_spec
    from zinfer_b200.engine.model import declared_tensors

    raw = U.CONFIGS["mix"]
    fam = family_for(raw)
    assert fam.name == "Kesitar" and fam.config_class is KesitarConfig
    cfg = KesitarConfig.from_dict(raw)
    assert KesitarConfig.from_dict(cfg.to_dict()) == cfg                      # survives a round trip
    # the tensors the model asks for are exactly the design's names and shapes (the head is the embedding's table)
    for name, other in {**U.CONFIGS, **U.MECHANISMS}.items():
        declared = declared_tensors(kesitar_model_spec(KesitarConfig.from_dict(other)))
        want = U.tensor_shapes(other)
        assert {k for k, s in declared.items() if not s.optional} == set(want), name
        assert all(declared[k].shape == want[k] for k in want), name
    bare = copy.deepcopy(raw)
    del bare["embedding"], bare["logit_scale"]
    cfg = KesitarConfig.from_dict(bare)
    assert cfg.embedding_scale == 1.0 and cfg.logit_scale == 1.0
    for change, match in ((lambda c: c["layers"][0].__setitem__("type", "convolution"), "unknown mixer"),
                          (lambda c: c["layers"][1]["mixer"].__setitem__("kv_heads", 3), "do not divide"),
                          (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 18), "even and at most"),
                          (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("pool", 0), "pool"),
                          (lambda c: c["layers"][1]["mixer"]["mask"].pop("size"), "size"),
                          (lambda c: c["layers"][3]["mixer"].__setitem__("vdim", 8), "v_mix"),
                          (lambda c: c["layers"][0]["mixer"].pop("vdim"), "vdim"),
                          (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "unknown feed-forward"),
                          (lambda c: c["norm"].pop("eps"), "eps")):
        bad = copy.deepcopy(raw)
        change(bad)
        with pytest.raises(ConfigError, match=match):
            KesitarConfig.from_dict(bad)


def test_command_line_inspects_the_model(tmp_path):
    from zinfer_b200 import cli

    d = U.write_model(str(tmp_path / "m"), U.CONFIGS["mix"], U.make_weights(U.CONFIGS["mix"], seed=1))
    out = io.StringIO()
    assert cli.run(["inspect-config", d], out) == 0
    text = out.getvalue()
    assert "architecture: Kesitar" in text and "embedding_scale: 3.0" in text and "logit_scale: 0.7" in text
    assert "layer 0: hgrn2 (heads=3 dim=8 vdim=12); feed-forward: dense ff=40" in text
    assert "window=9 pooled blocks of 4 mixed values); feed-forward: dense ff=72" in text and "layer 2: hgrn2" in text
    assert "feed-forward: none" in text
    out = io.StringIO()
    assert cli.run(["inspect-weights", d], out) == 0 and "tensor_count:" in out.getvalue()


def test_caches_of_tokens_and_of_blocks():
    from zinfer_b200.config import KesitarConfig, kesitar_model_spec
    from zinfer_b200.engine import DecoderModel

    model = DecoderModel(kesitar_model_spec(KesitarConfig.from_dict(U.CONFIGS["mix"])), torch.float32, "cpu")
    kv, state = model.cache_needs()
    assert set(state) == {"run0", "run2"} and state["run0"].shape == (3, 8, 12) and state["run0"].dtype == torch.float32
    assert set(kv) == {"run1.tokens", "run1.pooled", "run3.tokens", "run3.pooled", "run4"}
    # tokens stay for the window, or until their block is complete where a block is longer than the window
    assert (kv["run1.tokens"].window, kv["run3.tokens"].window, kv["run4"].window) == (9, 7, 6)
    assert (kv["run1.pooled"].window, kv["run1.pooled"].tokens_per_entry, kv["run3.pooled"].tokens_per_entry) == (None, 4, 7)
    assert (kv["run1.tokens"].head_dim, kv["run1.tokens"].value_dim, kv["run1.pooled"].value_dim) == (16, 24, 24)


def test_pages_of_blocks_in_the_cache_manager():
    """One entry per several tokens: places appear with a block's last token, pages with the first entry they hold;
    nothing is given back before the request ends; the token pages go back behind the window."""
    from zinfer_b200.cache import CacheManager, OutOfPages, bytes_per_page, pages_for
    from zinfer_b200.cache.sizing import entry_pages
    from zinfer_b200.parts import KVCacheNeed

    needs = {"t": KVCacheNeed(1, 8, window=5), "p": KVCacheNeed(1, 8, tokens_per_entry=3)}
    m = CacheManager(needs, [], 4, 16, 2)
    assert [g.pool.num_pages for g in m.groups] == [16, entry_pages(16, 3, 2)] and entry_pages(16, 3, 2) == 8
    m.add_request("a")
    m.reserve("a", 2)
    assert m.block_table("a", 1) == [] and m.room("a") == min(16 * 4, (8 * 4 + 1) * 3 - 1)
    m.commit("a", 2)
    m.reserve("a", 1)
    assert len(m.block_table("a", 1)) == 1                       # the third token completes the first entry
    m.commit("a", 1)
    for _ in range(30):
        m.reserve("a", 1)
        m.commit("a", 1)
    assert m.length("a") == 33 and len(m.block_table("a", 1)) == 3 and -1 not in m.block_table("a", 1)   # 11 entries in 3 pages
    assert m.block_table("a", 0)[:7] == [-1] * 7                 # positions 0..27 have left the window of the next query
    assert m.slots_for("a", 1, 10, 1) == [m.block_table("a", 1)[2] * 4 + 2]
    m.add_request("b")
    assert m.can_reserve("b", 40) and not m.can_reserve("b", 61) and m.room("b") < 61
    with pytest.raises(OutOfPages):
        m.reserve("b", 200)
    m.check()
    m.free_request("a")
    m.free_request("b")
    assert m.groups[1].pool.num_used == 0
    m.check()
    # a budget: a page of tokens costs its own bytes and a third of a page of entries
    assert bytes_per_page(needs, 4, 2) == 4 * 16 * 2 + -(-4 * 16 * 2 // 3)
    assert pages_for(needs, 4, 2, tokens=33, requests=2) == 9
    per_page, extra = bytes_per_page(needs, 4, 2), 3 * 4 * 16 * 2
    assert pages_for(needs, 4, 2, budget_bytes=10 * per_page + extra, requests=2) == 10
    with pytest.raises(ValueError):
        CacheManager({"x": KVCacheNeed(1, 8, window=5, tokens_per_entry=2)}, [], 4, 16, 2)


def test_step_arrays_of_blocks():
    """The step builder's places for entries: only the token that completes a block has one."""
    from zinfer_b200.cache import CacheManager
    from zinfer_b200.engine.batch import StepEntry, build_step
    from zinfer_b200.parts import KVCacheNeed

    m = CacheManager({"t": KVCacheNeed(1, 8, window=6), "p": KVCacheNeed(1, 8, tokens_per_entry=3)}, [], 4, 16, 3)
    for rid, have in (("a", 5), ("b", 0)):
        m.add_request(rid)
        if have:
            m.reserve(rid, have)
            m.commit(rid, have)
    m.reserve_all(["a", "b"], [8, 2])
    ctx = build_step(m, [StepEntry("a", list(range(8))), StepEntry("b", [1, 2])], "cpu", 16)
    got = ctx.kv_groups[1].slot_mapping.tolist()
    table = m.block_table("a", 1)
    # request a brings positions 5..12: 5, 8 and 11 complete entries 1, 2 and 3
    assert got == [table[0] * 4 + 1, -1, -1, table[0] * 4 + 2, -1, -1, table[0] * 4 + 3, -1, -1, -1]
    assert ctx.kv_groups[1].block_tables.tolist()[0][0] == table[0] and ctx.kv_groups[1].block_tables.tolist()[1][0] == -1
    assert (ctx.kv_groups[0].slot_mapping >= 0).all()


def test_weights_that_do_not_fit_are_refused(tmp_path):
    from zinfer_b200.engine import ModelRunner

    cfg = U.CONFIGS["odd"]
    for change, match in ((lambda w: w.__setitem__("l1.mix.lower", torch.zeros(7, dtype=torch.bfloat16)), "l1.mix.lower"),
                          (lambda w: w.pop("l0.norm2b"), "l0.norm2b"), (lambda w: w.pop("l0.mix.vmix"), "l0.mix.vmix"),
                          (lambda w: w.__setitem__("l0.mix.o.b", torch.zeros(43, dtype=torch.bfloat16)), "l0.mix.o.b")):
        w = U.make_weights(cfg, seed=2)
        change(w)
        d = U.write_model(str(tmp_path / "bad"), cfg, w)
        with pytest.raises(Exception, match=match):
            ModelRunner.from_model_dir(d, dtype=torch.float32, device="cpu", page_size=8, max_tokens=64, max_requests=2,
                                       cuda_graphs=False)


@pytest.mark.parametrize("name", ["mix", "alt", "odd"])
def test_engine_host_logic_on_stand_ins(cpu_kernels, tmp_path, name):
    cfg = U.CONFIGS[name]
    weights = U.make_weights(cfg, seed=3)
    runner = make_runner(tmp_path, cfg, weights, torch.float32, "cpu", max_tokens=192, max_requests=3, cuda_graphs=False)
    reqs = ru.make_requests(cfg["vocab"], [23, 1, 40, 9, 17], seed=4)
    plain = U.plain_logits(cfg, weights, reqs)
    for mode, trace in (("whole", ru.trace_whole(reqs)), ("tail", ru.trace_tail_decode(reqs, 6)),
                        ("portions", ru.trace_portions(reqs, 2)), ("mixed", ru.trace_mixed(reqs, 5, max_live=3, tail=4))):
        got = ru.run_in_process(runner, trace)
        ru.assert_close(got, plain, what=f"{name}/{mode}", argmax_frac=0.0, rtol=2e-4, atol=1e-5)
        assert not runner.manager.requests
    assert runner.manager.slots.reused > 0            # three slots served five requests, four times over


def test_greedy_generation_on_stand_ins(cpu_kernels, tmp_path):
    """Scheduler and entry point with a pool that is too small for all requests at once: preemption and recomputation
    give the tokens that each request gives alone."""
    from zinfer_b200.engine.api import Engine
    from zinfer_b200.sampling import SamplingParams

    cfg = U.MECHANISMS["blocks"]
    weights = U.make_weights(cfg, seed=5)
    d = U.write_model(str(tmp_path / "gen"), cfg, weights)
    prompts = list(ru.make_requests(cfg["vocab"], [11, 20, 3], seed=8).values())
    outs = []
    for tokens in (160, 40):
        eng = Engine(d, dtype="float32", device="cpu", page_size=4, kv_cache_tokens=tokens, max_batched_tokens=8, max_requests=3)
        outs.append([r.token_ids for r in eng.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=12, ignore_eos=True))])
    assert outs[0] == outs[1] and all(len(t) == 12 for t in outs[0])


def test_plain_model_pieces():
    """The plain implementation against numbers worked out by hand."""
    F = torch.float64
    # layer norm: (1, 3) has mean 2 and variance 1
    assert torch.allclose(P.layer_norm(torch.tensor([[1.0, 3.0]], dtype=F), torch.tensor([2.0, 5.0], dtype=F), 0.0), torch.tensor([[-2.0, 5.0]], dtype=F))
    assert torch.allclose(P.layer_norm(torch.tensor([[1.0, 3.0]], dtype=F), torch.ones(2, dtype=F), 3.0), torch.tensor([[-0.5, 0.5]], dtype=F))
    assert torch.allclose(P.rms_norm(torch.tensor([[3.0, 4.0]], dtype=F), torch.tensor([1.0, 2.0], dtype=F), 0.0), torch.tensor([[3.0, 8.0]], dtype=F) / 12.5 ** 0.5)
    # rotation: the second pair of four dimensions rotates by position * base^(-2/4); the fifth passes
    r = P.rotate(torch.tensor([[[0.0, 1.0, 0.0, 0.0, 9.0]]], dtype=F), torch.tensor([3]), {"dims": 4, "base": 16.0})
    assert torch.allclose(r, torch.tensor([[[0.0, np.cos(0.75), 0.0, np.sin(0.75), 9.0]]], dtype=F))
    # a window of 3 with blocks of 2 at position 7: tokens 5, 6, 7; block 1 (2, 3) is seen, block 2 (4, 5) is not
    mask = {"size": 3, "pool": 2}
    assert [j for j in range(10) if P.token_visible(7, j, mask)] == [5, 6, 7]
    assert [b for b in range(5) if P.block_visible(7, b, mask)] == [0, 1] and [b for b in range(5) if P.block_visible(8, b, mask)] == [0, 1, 2]
    assert torch.allclose(P.pooled(torch.arange(5.0, dtype=F).view(5, 1, 1), 2).flatten(), torch.tensor([0.5, 2.5], dtype=F))
    # softmax with a sink: two keys of score 0 and the sink share the weight
    out = P.attend(torch.zeros(1, 1, dtype=F), torch.zeros(2, 1, 1, dtype=F), torch.tensor([[[3.0]], [[6.0]]], dtype=F), torch.tensor([True, True]), 1.0, 1.0)
    assert torch.allclose(out, torch.tensor([[3.0]], dtype=F))
    assert torch.allclose(P.mix_values(torch.tensor(1.0), torch.tensor(5.0), 0.25), torch.tensor(2.0))
    # the forget gate: sigmoid(0) = 1/2 between the lower bound and 1; the state takes 1 - f of the value
    assert torch.allclose(P.forget_gate(torch.zeros(1, dtype=F), torch.tensor([0.2], dtype=F)), torch.tensor([0.6], dtype=F))
    one = torch.ones(1, 1, dtype=F)
    p = {"q": one, "f": 0 * one, "f.b": torch.zeros(1), "lower": torch.tensor([0.2]), "v": 3 * one, "norm": torch.ones(1), "o": one}
    _, S = P.hgrn2(torch.ones(2, 1, dtype=F), p, {"heads": 1, "dim": 1, "vdim": 1}, None, 0.0)
    assert torch.allclose(S, torch.tensor([[[0.6 * 1.2 + 0.4 * 3.0]]], dtype=F), atol=1e-6)


# ============================================================================ GPU
gpu = pytest.mark.gpu


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(U.MECHANISMS))
def test_each_mechanism_alone(tmp_path, name, dtype):
    cfg = U.MECHANISMS[name]
    weights = U.make_weights(cfg, seed=11)
    reqs = ru.make_requests(cfg["vocab"], [37, 1, 20], seed=12)
    plain = U.plain_logits(cfg, weights, reqs)
    runner = make_runner(tmp_path, cfg, weights, dtype, DEV, max_tokens=128, max_requests=2)
    for mode, trace in (("whole", ru.trace_whole(reqs)), ("tail", ru.trace_tail_decode(reqs, 12)),
                        ("portions", ru.trace_portions(reqs, 7, sizes=(2, 1, 5, 2, 3, 9, 2)))):
        got = ru.run_in_process(runner, trace)
        ru.assert_close(got, plain, what=f"{name}/{mode}", argmax_frac=0.0, **TOL[dtype])
    runner.manager.check()


@pytest.fixture(scope="module")
def models():
    """Per configuration: weights, requests, the plain model's logits."""
    out = {}
    for name, cfg in U.CONFIGS.items():
        weights = U.make_weights(cfg, seed=21 + len(name))
        reqs = ru.make_requests(cfg["vocab"], [45, 3, 70, 18, 1, 33], seed=5)
        out[name] = (cfg, weights, reqs, U.plain_logits(cfg, weights, reqs))
    return out


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(U.CONFIGS))
def test_whole_decode_portions_mixed(tmp_path, models, name, dtype):
    cfg, weights, reqs, plain = models[name]
    # pool: the three longest requests rounded up to pages, so pages and the three slots are used again
    runner = make_runner(tmp_path, cfg, weights, dtype, DEV, max_tokens=176, max_requests=3, poison_freed_pages=True)
    for mode, trace in (("whole", ru.trace_whole(reqs)), ("tail", ru.trace_tail_decode(reqs, 24)),
                        ("portions", ru.trace_portions(reqs, 9)), ("mixed", ru.trace_mixed(reqs, 13, max_live=3, tail=10))):
        got = ru.run_in_process(runner, trace)
        ru.assert_close(got, plain, what=f"{name}/{mode}", argmax_frac=0.0, **TOL[dtype])
        assert not runner.manager.requests
    assert runner.graphs is not None and runner.graphs.replays > 0         # single tokens came from CUDA graphs
    assert all(g.pool.reused > 0 for g in runner.manager.groups)           # pages of tokens and pages of blocks
    assert runner.manager.slots.reused > 0
    runner.manager.check()


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_batch_against_each_alone(tmp_path, models, dtype):
    """Unequal requests in one batch give the rows they give alone, to the last bits in float32."""
    from zinfer_b200.engine import StepEntry

    cfg, weights, reqs, _ = models["mix"]
    runner = make_runner(tmp_path, cfg, weights, dtype, DEV, max_tokens=256, max_requests=4)
    ids = ["r0", "r2", "r3", "r4"]
    alone = {}
    for rid in ids:
        alone[rid] = runner.step([StepEntry(rid, reqs[rid], list(range(len(reqs[rid]))))]).clone()
        runner.end_request(rid)
    half = len(reqs["r0"]) // 2
    runner.step([StepEntry("r0", reqs["r0"][:half], [])])
    entries = [StepEntry("r0", reqs["r0"][half:], list(range(len(reqs["r0"]) - half)))] + \
        [StepEntry(rid, reqs[rid], list(range(len(reqs[rid])))) for rid in ids[1:]]
    got = runner.step(entries)
    row = 0
    for e in entries:
        want = alone[e.request_id][-len(e.want):]
        part = got[row:row + len(e.want)]
        row += len(e.want)
        tol = 2e-6 if dtype == torch.float32 else 2e-2
        assert (part - want).abs().max() <= tol * want.abs().max(), e.request_id


# ---------------------------------------------------------------- edges of windows and blocks, the sink, far blocks
# one layer only: the tolerance in bfloat16 is tighter, so that a block one token early or late shows
EDGE_TOL = {torch.float32: TOL[torch.float32], torch.bfloat16: dict(rtol=2.5e-2, atol=4e-3)}


def _peaky(mixer, width=64, vocab=149, seed=31):
    """One attention layer without a feed-forward whose update weighs three times as much as the embedding, and whose
    queries all point much the same way (a large bias, nothing along the rotated dimensions), so that some tokens' keys
    are loud for every query and the rest are quiet."""
    cfg = U.config(vocab, width, [U.layer("attention", mixer)])
    w = U.make_weights(cfg, seed=seed)
    w["l0.norm1b"] = (w["l0.norm1b"].float() * 3.0).to(torch.bfloat16)
    rot = mixer.get("rot", {"dims": 0})["dims"]
    q, b = w["l0.mix.q"].float().view(mixer["heads"], -1, width), w["l0.mix.q.b"].float().view(mixer["heads"], -1)
    g = torch.Generator().manual_seed(seed)
    b = torch.randn(mixer["kv_heads"], b.shape[1], generator=g).repeat_interleave(mixer["heads"] // mixer["kv_heads"], 0) * 4.0 + 0.3 * b
    q[:, :rot] *= 0.2
    b[:, :rot] *= 0.05
    w["l0.mix.q"], w["l0.mix.q.b"] = (t.reshape(n.shape).to(torch.bfloat16) for t, n in ((q, w["l0.mix.q"]), (b, w["l0.mix.q.b"])))
    return cfg, w


def _loud_requests(cfg, weights, lengths, seed, only=None):
    """Requests of quiet tokens with a block of a loud one here and there (all of the block but its last token, where it
    has several): whether that block, or a loud token at the window's edge, is seen decides the output.  ``only``: one
    such block, of this number, all of it loud."""
    m = cfg["layers"][0]["mixer"]
    p = P._sub(weights, "l0.mix.")
    h = P.layer_norm(weights["embed"].double(), weights["l0.norm1"], 1e-5)
    k, _ = P.attention_cache(h, p, {**m, "rot": None}, 0, 1e-5, {})
    q = P.rms_norm((h @ p["q"].double().T + p["q.b"].double()).view(-1, m["heads"], m["dim"]), p["q.norm"], 1e-5).mean(0)
    loudness = torch.einsum("hd,nhd->nh", q, k.repeat_interleave(m["heads"] // m["kv_heads"], 1)).mean(-1)
    order = loudness.argsort(descending=True).tolist()
    loud, quiet = order[:8], order[len(order) // 2:]
    rng = np.random.default_rng(seed)
    pool, window = m["mask"].get("pool", 1), m["mask"]["size"]
    reqs = {}
    for r, n in enumerate(lengths):
        toks = [int(rng.choice(quiet)) for _ in range(n)]
        b, nth = 1, int(rng.integers(8))
        if only is not None:
            toks[only * pool:(only + 1) * pool] = [loud[0]] * pool
            b = n
        while (b + 1) * pool <= n:
            for j in range(max(1, pool - 1)):
                toks[b * pool + j] = loud[nth % len(loud)]
            nth += 1
            b += max(2, (window + 3) // pool)
        reqs[f"r{r}"] = toks
    return reqs


EDGES = {
    # windows and blocks that end inside pages, at their edges and beyond several of them
    "small": U.att(4, 2, 16, 24, 0.8, window=21, pool=5, rot=(4, 100.0)),
    "block_longer_than_window": U.att(2, 1, 16, 8, 0.8, window=7, pool=18),
    "block_of_a_page": U.att(4, 1, 64, 64, 0.35, window=32, pool=16, rot=(32, 1000.0)),
    "tensor_sizes": U.att(4, 2, 128, 128, 0.35, window=50, pool=7, rot=(32, 100.0)),
    "narrow_values": U.att(4, 2, 64, 24, 0.4, window=29, pool=3, rot=(16, 100.0)),
    "narrow_keys": U.att(6, 1, 40, 96, 0.8, window=33, pool=2),
}


def _wrong(cfg, weights, reqs):
    """The plain model's logits with a window or a block's visibility one off either way, without blocks, and with sums
    of blocks in place of their means: what an engine with that fault would give."""
    out, right_t, right_b, right_p = {}, P.token_visible, P.block_visible, P.pooled
    shifted = lambda mask, by: {**mask, "size": mask["size"] + by}
    try:
        for what, by in (("window one too wide", 1), ("window one too narrow", -1)):
            P.token_visible = lambda i, j, mask, by=by: right_t(i, j, shifted(mask, by))
            out[what] = U.plain_logits(cfg, weights, reqs)
        P.token_visible = right_t
        for what, by in (("block one token early", -1), ("block one token late", 1)):
            P.block_visible = lambda i, b, mask, by=by: right_b(i, b, shifted(mask, by))
            out[what] = U.plain_logits(cfg, weights, reqs)
        P.block_visible = lambda i, b, mask: False
        out["no blocks"] = U.plain_logits(cfg, weights, reqs)
        P.block_visible = right_b
        P.pooled = lambda keys, n: right_p(keys, n) * n
        out["sums for means"] = U.plain_logits(cfg, weights, reqs)
    finally:
        P.token_visible, P.block_visible, P.pooled = right_t, right_b, right_p
    return out


@pytest.mark.parametrize("case", list(EDGES))
def test_the_peaky_requests_show_every_fault_of_the_mask(case):
    """The plain model alone: with the window or a block's visibility one off, the logits move by more than the loosest
    tolerance of the tests below at many positions."""
    cfg, weights = _peaky(EDGES[case])
    reqs = _loud_requests(cfg, weights, [170], seed=6)
    plain = U.plain_logits(cfg, weights, reqs)
    for what, other in _wrong(cfg, weights, reqs).items():
        moved = np.abs(other["r0"] - plain["r0"]).max(axis=-1) / np.abs(plain["r0"]).max(axis=-1)
        assert (moved > 2 * EDGE_TOL[torch.bfloat16]["rtol"]).sum() >= 2, (what, np.sort(moved)[-5:])


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", list(EDGES))
def test_every_edge_of_windows_and_blocks_decides(tmp_path, dtype, case):
    """Prompts of a few hundred tokens with peaky attention (the test above shows that each fault of the mask moves
    these logits by far more than the tolerance): whole, in portions that end around the edges of pages, windows and
    blocks, decoding token by token far past the window (so that pages leave it and are used again), and mixed."""
    mixer = EDGES[case]
    cfg, weights = _peaky(mixer)
    window, pool = mixer["mask"]["size"], mixer["mask"]["pool"]
    page = 16
    n = 3 * window + 70
    reqs = _loud_requests(cfg, weights, [n, window + pool + 2, window, 3], seed=6)
    plain = U.plain_logits(cfg, weights, reqs)
    runner = make_runner(tmp_path, cfg, weights, dtype, DEV, page_size=page, max_tokens=2 * (n + page) + 4 * page,
                         max_requests=3, poison_freed_pages=True)
    edges = (page, page - 1, 1, pool, 2 * page - 1, 2, window, 2, window - 1, 3, pool + 1, 1, 1, 5, max(1, pool - 1), 2, 40)
    for mode, trace in (("whole", ru.trace_whole(reqs)), ("edges", ru.trace_portions(reqs, 0, sizes=edges)),
                        ("long decode", ru.trace_tail_decode(reqs, 2 * window + 30)),
                        ("mixed", ru.trace_mixed(reqs, 3, max_live=3, tail=window + 9))):
        got = ru.run_in_process(runner, trace)
        ru.assert_close(got, plain, what=f"edges {case}/{mode}", argmax_frac=0.0, **EDGE_TOL[dtype])
    assert runner.graphs is not None and runner.graphs.replays > window
    assert sum(g.pool.reused for g in runner.manager.groups) > 0
    runner.manager.check()


@gpu
@pytest.mark.parametrize("page", [4, 8, 24, 64])
def test_other_page_sizes(tmp_path, page):
    """Pages smaller than a block, larger than the window, and no power of two, on both attention kernels."""
    for case in ("small", "tensor_sizes"):
        cfg, weights = _peaky(EDGES[case])
        reqs = _loud_requests(cfg, weights, [150, 40], seed=16)
        plain = U.plain_logits(cfg, weights, reqs)
        runner = make_runner(tmp_path, cfg, weights, torch.bfloat16, DEV, page_size=page, max_tokens=256, max_requests=2, poison_freed_pages=True)
        for mode, trace in (("whole", ru.trace_whole(reqs)), ("tail", ru.trace_tail_decode(reqs, 30)),
                            ("mixed", ru.trace_mixed(reqs, 3, max_live=2, tail=20))):
            ru.assert_close(ru.run_in_process(runner, trace), plain, what=f"page {page} {case}/{mode}", argmax_frac=0.0, **EDGE_TOL[torch.bfloat16])


@gpu
def test_the_sink_carries_the_first_tokens(tmp_path):
    """Where scores are low the sink holds much of the softmax's denominator at a sequence's first tokens: the plain model
    without it gives other logits by far, and the engine matches the one with it.  (The norm of the layer's output
    would undo a factor common to all heads, so one head's scores are made low and the other's high.)"""
    for d in (8, 64):
        cfg = U.config(61, 32, [U.A(2, 2, d, d, 8.0 / d, window=4, pool=3)])
        weights = U.make_weights(cfg, seed=31)
        weights["l0.norm1b"] = (weights["l0.norm1b"].float() * 3.0).to(torch.bfloat16)
        for n in ("q", "k"):
            weights[f"l0.mix.{n}"][:d] *= 0.2
            weights[f"l0.mix.{n}.b"][:d] = 0.05 if n == "k" else -0.05
            weights[f"l0.mix.{n}.b"][d:] = 6.0
        weights["l0.mix.q.norm"][:] = 0.5
        reqs = ru.make_requests(cfg["vocab"], [12, 2, 1], seed=9)
        plain = U.plain_logits(cfg, weights, reqs)
        no_sink = U.plain_logits(cfg, weights, reqs, sink=0.0)
        assert all(np.abs(plain[r] - no_sink[r]).max() > 0.15 * np.abs(plain[r]).max() for r in reqs)
        for dtype in (torch.float32, torch.bfloat16):
            runner = make_runner(tmp_path, cfg, weights, dtype, DEV, max_tokens=64, max_requests=2)
            for trace in (ru.trace_whole(reqs), ru.trace_tail_decode(reqs, 11), ru.trace_portions(reqs, 3, sizes=(2, 1, 2, 3))):
                ru.assert_close(ru.run_in_process(runner, trace), plain, what="sink", argmax_frac=0.0, **EDGE_TOL[dtype])


def _far_block():
    cfg, weights = _peaky(U.att(2, 1, 16, 12, 0.9, window=10, pool=2, rot=(2, 100.0)))
    toks = _loud_requests(cfg, weights, [270], seed=7, only=9)["r0"]
    return cfg, weights, toks


def test_the_far_block_matters():
    """In the plain model the last positions' logits are others without the one loud block 250 tokens back."""
    cfg, weights, toks = _far_block()
    right = P.Plain(cfg, weights).forward(toks)[-5:].numpy()
    lost = P.Plain(cfg, weights).forward(toks[:18] + toks[16:18] + toks[20:])[-5:].numpy()
    assert (np.abs(right - lost).max(-1) > 0.2 * np.abs(right).max(-1)).all()


@gpu
def test_a_single_far_block_decides(tmp_path):
    """One block of tokens hundreds of positions back carries much of the last queries' softmax (the test above); an
    engine that lost that block could not match."""
    cfg, weights, toks = _far_block()
    plain = U.plain_logits(cfg, weights, {"r0": toks})
    for dtype in (torch.float32, torch.bfloat16):
        runner = make_runner(tmp_path, cfg, weights, dtype, DEV, page_size=16, max_tokens=288, max_requests=1)
        for trace in (ru.trace_whole({"r0": toks}), ru.trace_tail_decode({"r0": toks}, 5)):
            ru.assert_close(ru.run_in_process(runner, trace), plain, what="one far block", argmax_frac=0.0, **TOL[dtype])


@gpu
def test_a_state_that_remembers(tmp_path):
    """Forget gates close to 1: what a sequence's first token wrote still shows hundreds of tokens later, through many
    portions, and a request that takes a used slot starts from nothing."""
    cfg = U.config(83, 48, [U.H(2, 16, 16)])
    weights = U.make_weights(cfg, seed=41)
    weights["l0.mix.lower"][:] = 0.99
    weights["l0.mix.f.b"][:] = 4.0
    weights["l0.norm1b"] = (weights["l0.norm1b"].float() * 3.0).to(torch.bfloat16)
    toks = ru.make_requests(cfg["vocab"], [300], seed=7)["r0"]
    reqs = {"r0": toks, "r1": [(toks[0] + 40) % 83] + toks[1:], "r2": toks[:3]}
    plain = U.plain_logits(cfg, weights, reqs)
    moved = np.abs(plain["r0"][200:] - plain["r1"][200:]).max(-1) / np.abs(plain["r0"][200:]).max(-1)
    assert moved.min() > 20 * TOL[torch.float32]["rtol"]                   # the first token still shows at every one
    for dtype in (torch.float32, torch.bfloat16):
        runner = make_runner(tmp_path, cfg, weights, dtype, DEV, max_tokens=320, max_requests=1)
        for trace in (ru.trace_whole(reqs), ru.trace_tail_decode(reqs, 250), ru.trace_portions(reqs, 3)):
            ru.assert_close(ru.run_in_process(runner, trace), plain, what="memory", argmax_frac=0.0, **TOL[dtype])


REAL = U.config(257, 256, [
    U.H(4, 64, 64, ff=384),
    U.A(4, 2, 64, 64, 0.12, window=40, pool=8, rot=(32, 10000.0), v_mix=True, ff=320),
    U.H(2, 128, 128, ff=128),
    U.A(2, 1, 128, 128, 0.09, window=90, pool=16, rot=(128, 10000.0)),
    U.A(8, 2, 96, 64, 0.1, window=64, pool=5, rot=(64, 10000.0), v_mix=True, ff=128),
    U.A(8, 2, 64, 64, 0.1, v_mix=True),
], embed_scale=5.0, logit_scale=0.3)


@gpu
def test_sizes_of_a_real_layer(tmp_path):
    """Heads of 64, 96 and 128, rows the tensor-core products take: the fast kernels against the plain model, in prompts of
    a few hundred tokens, decoded tails and mixed batches."""
    weights = U.make_weights(REAL, seed=71)
    reqs = ru.make_requests(REAL["vocab"], [230, 37, 120, 5], seed=5)
    plain = U.plain_logits(REAL, weights, reqs)
    for dtype in (torch.float32, torch.bfloat16):
        runner = make_runner(tmp_path, REAL, weights, dtype, DEV, page_size=16, max_tokens=480, max_requests=3, poison_freed_pages=True)
        for mode, trace in (("whole", ru.trace_whole(reqs)), ("tail", ru.trace_tail_decode(reqs, 90)),
                            ("portions", ru.trace_portions(reqs, 4, sizes=(33, 2, 64, 17, 1, 40))),
                            ("mixed", ru.trace_mixed(reqs, 2, max_live=3, tail=20))):
            ru.assert_close(ru.run_in_process(runner, trace), plain, what=f"real sizes/{mode}", argmax_frac=0.0, **TOL[dtype])
        runner.manager.check()
        if dtype == torch.bfloat16:
            # a prompt and a single token ran on the tensor-core kernels, not on the exact ones
            from zinfer_b200 import profiling
            from zinfer_b200.engine import StepEntry
            with profiling.profile() as prof:
                runner.step([StepEntry("p", reqs["r0"][:200], [199])])
                runner.step([StepEntry("p", reqs["r0"][200:201], [0])])
            runner.end_request("p")
            ran = {c["class"] for c in prof.summary()["classes"]}
            assert {"attention (prefill, mma.sync, pooled blocks)", "attention (decode, pooled blocks)"} <= ran, ran
            assert "attention (exact, CUDA cores)" not in ran, ran


@gpu
def test_fast_kernels_agree_with_the_exact_ones(tmp_path, monkeypatch):
    """The same bfloat16 model on the tensor-core attention kernels and on the exact kernels: whole prompts, portions
    and single tokens agree to the rounding of the softmax weights' second part."""
    from zinfer_b200 import ops

    cfg = U.config(131, 128, [
        U.A(8, 2, 64, 64, 0.25, window=70, pool=12), U.A(4, 4, 128, 128, 0.2, window=33, pool=1, rot=(64, 100.0)),
        U.A(16, 1, 72, 40, 0.2, window=64, pool=20), U.A(20, 2, 128, 56, 0.2, window=17, pool=3, v_mix=True), U.A(2, 1, 32, 56, 0.3),
    ])
    weights = U.make_weights(cfg, seed=81)
    reqs = ru.make_requests(cfg["vocab"], [400, 130, 33], seed=2)
    traces = (ru.trace_whole(reqs), ru.trace_tail_decode(reqs, 20), ru.trace_portions(reqs, 5, sizes=(64, 3, 129, 32, 1, 40)),
              ru.trace_mixed(reqs, 4, max_live=3, tail=12))
    got = {}
    for backend in ("generic", "auto"):
        monkeypatch.setattr(ops, "ATTENTION_BACKEND", backend)
        runner = make_runner(tmp_path, cfg, weights, torch.bfloat16, DEV, page_size=16, max_tokens=640, max_requests=3)
        got[backend] = [ru.run_in_process(runner, t) for t in traces]
    for exact, fast in zip(got["generic"], got["auto"]):
        for key, row in exact.items():
            assert np.abs(fast[key] - row).max() <= 2e-2 * np.abs(row).max(), key


@gpu
def test_greedy_generation_through_the_engine(tmp_path, models):
    from zinfer_b200.engine.api import Engine
    from zinfer_b200.sampling import SamplingParams

    cfg, weights, reqs, _ = models["mix"]
    d = U.write_model(str(tmp_path / "gen"), cfg, weights)
    prompts = [reqs["r1"], reqs["r3"], reqs["r0"][:30], reqs["r4"]]
    eng = Engine(d, dtype="float32", device=DEV, page_size=8, kv_cache_tokens=192, max_batched_tokens=16, max_requests=3)
    got = eng.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=25, ignore_eos=True))
    for p, r in zip(prompts, got):
        assert len(r.token_ids) == 25                              # past the windows and several blocks
        logits = P.Plain(cfg, weights).forward(p + r.token_ids).numpy()
        for i, t in enumerate(r.token_ids):      # the best token given the same history, or tied with it to rounding
            row = logits[len(p) - 1 + i]
            assert row[t] >= row.max() - 1e-4 * np.abs(row).max()


@gpu
def test_command_line_makes_a_random_model_and_generates(tmp_path):
    """bin/zinfer: a model folder of random weights made from a Kesitar config.json, then tokens from it, greedy and sampled."""
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(U.CONFIGS["odd"]))
    d = str(tmp_path / "random")
    tool = os.path.join(ru.REPO, "bin", "zinfer")
    r = subprocess.run([sys.executable, tool, "random-model", d, str(cfg_path), "7"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    r = subprocess.run([sys.executable, tool, "generate-token-ids", d, "5,17,3,60,2", "6", "--dtype", "float32"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0 and "tokens: [5, 17, 3, 60, 2, " in r.stdout, r.stderr[-2000:]
    r = subprocess.run([sys.executable, tool, "generate-token-ids", d, "5,17,3,60,2", "6", "--temperature", "0.8", "--top-k", "10",
                        "--seed", "3"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0 and "tokens: [5, 17, 3, 60, 2, " in r.stdout, r.stderr[-2000:]


@gpu
def test_replay_program(tmp_path, models):
    """bin/trace_run as a user runs it: the model class comes from config.json, four state slots."""
    cfg, weights, reqs, plain = models["odd"]
    d = U.write_model(str(tmp_path / "tool"), cfg, weights)
    trace = ru.trace_mixed(reqs, 3, max_live=4, tail=8)
    info = {}
    got = ru.run_trace_tool(d, "float32", trace, str(tmp_path / "out"), ru.max_live_tokens(trace), cfg["vocab"], info=info)
    ru.assert_close(got, plain, what="trace_run", argmax_frac=0.0, **TOL[torch.float32])
    assert info["pages_reused"] and info["pages_reused"] > 0


# ------------------------------------------------------------------ the new kernels alone, against their plain stand-ins
class _N:
    def __init__(self, weight, eps, kind):
        self.weight, self.eps, self.kind = weight, eps, kind


@gpu
@pytest.mark.parametrize("width", [4096, 640, 43, 2052, 7, 10240])
def test_sandwich_norm_against_plain_arithmetic(width):
    """Both kinds of norm on either side, updates whole and as partial sums and none, few rows and many, picked rows; a
    stream whose mean is a thousand times its spread."""
    import kernel_refs as R
    from zinfer_b200 import ops

    if width == 10240:
        cases = [(3, torch.bfloat16), (600, torch.bfloat16)]
    else:
        cases = [(1, torch.bfloat16), (9, torch.float32), (530, torch.bfloat16), (530, torch.float32)]
    g = torch.Generator(device=DEV).manual_seed(5)
    rnd = lambda *shape: torch.randn(*shape, generator=g, device=DEV)
    for T, dtype in cases:
        w1, w2 = 1 + 0.3 * rnd(width), 1 + 0.3 * rnd(width)
        tol = dict(rtol=1e-2, atol=1e-2) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=2e-4)
        for post, pre in (("layer", "layer"), ("rms", "layer"), (None, "rms"), ("layer", None)):
            for form in ("whole", "whole16", "parts", "none", "picked"):
                if form == "none" and (post or not pre) or form == "picked" and not pre:
                    continue
                h0 = rnd(T, width) + (30.0 if pre == "layer" else 0.0)
                a = 2.0 * rnd(T, width) + 5.0
                if form == "whole16":
                    a = a.to(torch.bfloat16)
                da = ops.Partials(torch.stack([0.5 * a, 0.2 * a, 0.3 * a]).contiguous()) if form == "parts" else (None if form == "none" else a)
                rows = torch.tensor([T - 1, 0, T // 2, 0], dtype=torch.int32, device=DEV) if form == "picked" else None
                norm = _N(w1, 1e-3, post) if post else None
                h, hr = h0.clone(), h0.clone()
                got = ops.sandwich_norm(h, ops.PostNormed(da, norm) if norm else da, w2 if pre else None, 1e-5, pre or "rms", dtype, rows=rows)
                ra = None if form == "none" else a
                want = R.sandwich_norm(hr, R.PostNormed(ra, norm) if norm else ra, w2 if pre else None, 1e-5, pre or "rms", dtype, rows=rows)
                what = (width, T, dtype, post, pre, form)
                assert torch.allclose(h, hr, rtol=1e-5, atol=1e-4), what
                assert (got is None) == (want is None) and (got is None or torch.allclose(got.float(), want.float(), **tol)), what


@gpu
def test_head_rows_and_pooled_blocks_against_plain_arithmetic():
    """zi_qkv_heads_prepare and zi_pool_blocks: each against a few lines of PyTorch, rows whole and as partial sums, sizes
    that 16-byte accesses take and others."""
    import kernel_refs as R
    from zinfer_b200 import ops

    g = torch.Generator(device=DEV).manual_seed(6)
    rnd = lambda *shape: torch.randn(*shape, generator=g, device=DEV)
    page = 8
    for T, nq, nkv, d, dv, rot, dtype in ((5, 6, 2, 12, 20, 8, torch.bfloat16), (200, 4, 4, 64, 64, 64, torch.bfloat16),
                                          (33, 3, 1, 10, 7, 6, torch.float32), (40, 8, 2, 128, 48, 30, torch.bfloat16), (9, 2, 1, 16, 4, 0, torch.float32)):
        width = nq * d + nkv * (d + dv)
        proj, bias, qw, kw = rnd(T, width), 0.3 * rnd(width), 1 + 0.2 * rnd(d), 1 + 0.2 * rnd(d)
        cos, sin = ops.rope_table_freqs(300, torch.rand(max(1, rot // 2), generator=g, device=DEV), 1.0) if rot else (None, None)
        pos = torch.randint(0, 300, (T,), generator=g, device=DEV, dtype=torch.int32)
        slots = torch.randperm(40 * page, generator=g, device=DEV)[:T].to(torch.int32)
        slots[0] = -1                                                   # a row that pads a captured batch writes nothing
        first = rnd(T, nkv * dv)
        for src in (proj, ops.Partials(torch.stack([0.25 * proj, 0.75 * proj]).contiguous()), proj.to(torch.bfloat16)):
            if dtype == torch.float32 and not isinstance(src, ops.Partials) and src.dtype == torch.bfloat16:
                continue
            caches = [[torch.zeros(40, nkv, page, n, dtype=dtype, device=DEV) for n in (d, dv)] for _ in range(2)]
            tail = lambda c: (bias, nq, nkv, d, dv, qw, kw, 1e-5, rot, cos, sin, pos, *c, slots, page, dtype)
            got = ops.qkv_heads_prepare(src, *tail(caches[0]), mix_with=first, mix_lambda=0.3, keep_values=True)
            want = R.qkv_heads_prepare(proj if isinstance(src, ops.Partials) else src, *tail(caches[1]), mix_with=first, mix_lambda=0.3, keep_values=True)
            tol = dict(rtol=2e-2, atol=2e-2) if dtype == torch.bfloat16 else dict(rtol=2e-5, atol=2e-5)
            for a, b in zip((*got, *caches[0]), (*want, *caches[1])):
                assert torch.allclose(a.float(), b.float(), **tol)
            assert caches[0][0].abs().sum() > 0
        for per in (1, 3, 8, 11):
            class S:
                n_seqs, n_tokens = 2, 30
            S.cu_q = torch.tensor([0, 22, 30], dtype=torch.int32, device=DEV)
            S.positions = torch.cat([torch.arange(13, 35), torch.arange(0, 8)]).to(torch.int32).to(DEV)
            S.q_lens, S.ctx_lens = [22, 8], [13, 0]
            k, v = (rnd(12, nkv, page, n).to(dtype) for n in (d, dv))
            bt = torch.arange(10, dtype=torch.int32, device=DEV).view(2, 5)
            outs = []
            for mod in (ops, R):
                pk, pv = (torch.zeros(20, nkv, page, n, dtype=dtype, device=DEV) for n in (d, dv))
                entries = torch.tensor([(s * 9 + p // per // page) * page + (p // per) % page if (p + 1) % per == 0 else -1
                                        for s, p in [(0, p) for p in range(13, 35)] + [(1, p) for p in range(8)]], dtype=torch.int32, device=DEV)
                mod.pool_blocks(k, v, bt, mod.PooledKeys(pk, pv, None, per), entries, S, page)
                outs.append((pk.float(), pv.float()))
            assert all(torch.allclose(a, b, rtol=1e-2 if dtype == torch.bfloat16 else 1e-5, atol=1e-2 if dtype == torch.bfloat16 else 1e-5) for a, b in zip(*outs))
            assert outs[0][0].abs().sum() > 0


@gpu
def test_gated_recurrence_against_plain_arithmetic():
    """zi_linear_recurrence_gated: whole rows and partial sums, unequal requests, states carried, channels that are no power
    of two and more than one staging pass takes."""
    import kernel_refs as R
    from zinfer_b200 import ops

    g = torch.Generator().manual_seed(7)
    for heads, dim, vdim in ((3, 8, 12), (2, 48, 70), (1, 300, 20), (2, 128, 128), (4, 1, 3), (2, 33, 256), (1, 80, 64)):
        class S:
            n_seqs = 3
        S.cu_q = torch.tensor([0, 37, 38, 55], dtype=torch.int32)
        S.state_slots = torch.tensor([2, 0, 3], dtype=torch.int32)
        proj = torch.randn(55, heads * (2 * dim + vdim), generator=g)
        lower, bias = torch.rand(heads * dim, generator=g), torch.randn(heads * dim, generator=g)
        state0 = torch.randn(5, heads, dim, vdim, generator=g)
        ref_state = state0.clone()
        want = R.linear_recurrence_gated(proj, lower, bias, ref_state, heads, dim, vdim, S)
        D = type("D", (), {"n_seqs": 3, "cu_q": S.cu_q.to(DEV), "state_slots": S.state_slots.to(DEV)})
        p = proj.to(DEV)
        for src in (p, ops.Partials(torch.stack([0.5 * p, 0.25 * p, 0.25 * p]).contiguous())):
            state = state0.to(DEV)
            got = ops.linear_recurrence_gated(src, lower.to(DEV), bias.to(DEV), state, heads, dim, vdim, D)
            assert torch.allclose(got.cpu(), want, rtol=1e-4, atol=1e-3 * max(1.0, want.abs().max().item() / 10)), (heads, dim, vdim)
            assert torch.allclose(state.cpu(), ref_state, rtol=1e-4, atol=1e-4)
        # single tokens: where the sizes allow it one kernel, the head norm with it
        class One:
            n_seqs, all_decode = 5, True
            cu_q = torch.arange(6, dtype=torch.int32)
            state_slots = torch.tensor([2, 0, 3, 1, 4], dtype=torch.int32)
        w = 1 + 0.2 * torch.randn(vdim, generator=g)
        ref_state = state0.clone()
        want = R.linear_recurrence_gated(proj[:5], lower, bias, ref_state, heads, dim, vdim, One, norm_weight=w, norm_eps=1e-5)
        D = type("D", (), {"n_seqs": 5, "all_decode": True, "cu_q": One.cu_q.to(DEV), "state_slots": One.state_slots.to(DEV)})
        p = proj[:5].to(DEV)
        for src in (p, ops.Partials(torch.stack([0.5 * p, 0.25 * p, 0.25 * p]).contiguous())):
            for dtype in (torch.float32, torch.bfloat16):
                state = state0.to(DEV)
                got = ops.linear_recurrence_gated(src, lower.to(DEV), bias.to(DEV), state, heads, dim, vdim, D, norm_weight=w.to(DEV),
                                                  norm_eps=1e-5, out_dtype=dtype)
                tol = 1e-2 if dtype == torch.bfloat16 else 2e-4
                assert got.dtype == dtype and torch.allclose(got.float().cpu(), want, rtol=tol, atol=tol), (heads, dim, vdim)
                assert torch.allclose(state.cpu(), ref_state, rtol=1e-4, atol=1e-4)


@gpu
def test_recurrence_in_tiles_against_one_walk(tmp_path, monkeypatch):
    """Long portions cut into tiles that run side by side give what one walk over the portion gives: outputs and states,
    portions that end at a tile's edge and just beyond, beside single tokens and short portions, from states that earlier
    portions left; fast and slow forgetting."""
    from zinfer_b200 import ops
    from zinfer_b200.cache import CacheManager
    from zinfer_b200.engine.batch import StepEntry, build_step

    rows = ops.attention_prefill_tile_rows()
    g = torch.Generator(device=DEV).manual_seed(9)
    rnd = lambda *shape: torch.randn(*shape, generator=g, device=DEV)
    for heads, dim, vdim, lens in ((2, 16, 24, (2 * rows, 1, 5 * rows + 1, 2, 3 * rows - 1)), (1, 64, 64, (1, 1000)), (3, 300, 8, (2 * rows + 7,)),
                                   (2, 128, 128, (rows, 4 * rows, 1, rows + 1))):
        m = CacheManager({}, ["s"], 16, 1, 8)
        entries = []
        for i, n in enumerate(lens):
            m.add_request(i)
            entries.append(StepEntry(i, [0] * n))
        step = build_step(m, entries, DEV, ops.attention_tile_rows(), pf_tile_rows=rows)
        T = step.n_tokens
        proj = rnd(T, heads * (2 * dim + vdim))
        lower = 0.999 * torch.rand(heads * dim, generator=g, device=DEV)
        bias = 3.0 * rnd(heads * dim)
        w = 1 + 0.1 * rnd(vdim)
        state0 = rnd(9, heads, dim, vdim)
        outs = []
        for tiles in (False, True):
            monkeypatch.setattr(ops, "RECURRENCE_TILES", tiles)
            state = state0.clone()
            y = ops.linear_recurrence_gated(proj, lower, bias, state, heads, dim, vdim, step, norm_weight=w, norm_eps=1e-5, out_dtype=torch.bfloat16)
            outs.append((y.float(), state))
        assert torch.allclose(outs[0][1], outs[1][1], rtol=1e-4, atol=1e-4), (heads, dim, vdim)
        assert torch.allclose(outs[0][0], outs[1][0], rtol=2e-2, atol=2e-2), (heads, dim, vdim)
        assert not torch.equal(outs[1][1], state0)
