"""The Sumozen design in the engine against the plain implementation (tests/plain_sumozen.py).

Every test makes its own small configuration and weights (tests/sumozen_util.py).  The CPU tests put the plain
PyTorch stand-ins of the kernels (tests/kernel_refs.py) under the engine, so they test what is host logic:
configuration, registry, tensor names, caches and states per layer and branch, batching, scheduling.  The GPU tests run
the same traces on the kernels, in float32 and bfloat16: every mechanism alone, whole prompts, prompts followed by
token-by-token decoding (from CUDA graphs), portions down to one and two tokens, mixed batches of unequal requests with
pages and state slots that are used again, peaky attention across page edges, far keys, states that remember, the first
tokens of a sequence, and greedy generation through ``Engine.generate``.
"""
import copy
import io
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_sumozen as P
import replay_util as ru
import sumozen_util as U

DEV = "cuda:0"
# float32: the engine against 64-bit arithmetic, both from the same bfloat16-representable weights, relative to a
# row's largest logit.  bfloat16: products and activations are rounded to 8 bits of mantissa between kernels; the
# requests have no close calls of the routers (sumozen_util.clear_requests).
TOL = {torch.float32: dict(rtol=5e-5, atol=1e-6), torch.bfloat16: dict(rtol=6e-2, atol=4e-3)}


def make_runner(tmp_path, cfg, weights, dtype, device, **kw):
    from zinfer_b200.engine import ModelRunner

    d = U.write_model(str(tmp_path / f"m{abs(hash(json.dumps(cfg, sort_keys=True))) % 10**8}"), cfg, weights)
    kw.setdefault("page_size", 8)
    kw.setdefault("max_requests", 4)
    return ModelRunner.from_model_dir(d, dtype=dtype, device=device, **kw)


# ============================================================================ CPU
def test_config_is_read_and_registered():
    from zinfer_b200.config import ConfigError, SumozenConfig, family_for, sumozen_model_spec
    from zinfer_b200.engine.model import declared_tensors

    raw = U.CONFIGS["mix"]
    fam = family_for(raw)
    assert fam.name == "Sumozen" and fam.config_class is SumozenConfig
    cfg = SumozenConfig.from_dict(raw)
    assert SumozenConfig.from_dict(cfg.to_dict()) == cfg                      # survives a round trip
    for name, other in {**U.CONFIGS, **U.MECHANISMS}.items():
        declared = declared_tensors(sumozen_model_spec(SumozenConfig.from_dict(other)))
        want = U.tensor_shapes(other)
        assert {k for k, s in declared.items() if not s.optional} == set(want), name
        assert all(declared[k].shape == want[k] for k in want), name
    left = lambda c: c["layers"][0]["mixer"]["left"]
    for change, match in ((lambda c: c["layers"][0].__setitem__("type", "gla"), "unknown mixer"),
                          (lambda c: left(c).__setitem__("kv_heads", 3), "do not divide"),
                          (lambda c: left(c)["rot"].__setitem__("dims", 18), "even and at most"),
                          (lambda c: left(c)["rot"]["scaling"].pop("fast"), "fast"),
                          (lambda c: left(c).__setitem__("conv", 40), "taps"),
                          (lambda c: left(c).__setitem__("softcap", 0.0), "softcap"),
                          (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
                          (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
                          (lambda c: c["layers"][0]["mixer"]["right"].pop("vdim"), "vdim"),
                          (lambda c: c["layers"][1]["mixer"].__setitem__("groups", 4), "groups"),
                          (lambda c: c["layers"][1]["mixer"].__setitem__("norm_groups", 5), "norm groups"),
                          (lambda c: c["layers"][1]["mixer"].pop("state"), "state"),
                          (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "unknown feed-forward"),
                          (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 7), "cannot be chosen"),
                          (lambda c: c["norm"].pop("eps"), "eps")):
        bad = copy.deepcopy(raw)
        change(bad)
        with pytest.raises(ConfigError, match=match):
            SumozenConfig.from_dict(bad)


def test_command_line_inspects_the_model(tmp_path):
    from zinfer_b200 import cli

    d = U.write_model(str(tmp_path / "m"), U.CONFIGS["mix"], U.make_weights(U.CONFIGS["mix"], seed=1))
    out = io.StringIO()
    assert cli.run(["inspect-config", d], out) == 0
    text = out.getvalue()
    assert "architecture: Sumozen" in text and "layer 0: parallel (left 0.7 x attention (" in text and "softcap=6.0" in text
    assert "right 1.3 x delta rule (conv=4, dim=8, heads=4" in text and "moe experts=6 top=2 ff=40 shared ff=24" in text
    assert "layer 1: mamba2 (conv=4, groups=3, heads=6, norm_groups=2, state=16, vdim=8)" in text and "feed-forward: none" in text
    out = io.StringIO()
    assert cli.run(["inspect-weights", d], out) == 0 and "tensor_count:" in out.getvalue()


def test_caches_and_states_per_layer_and_branch():
    from zinfer_b200.config import SumozenConfig, sumozen_model_spec
    from zinfer_b200.engine import DecoderModel

    model = DecoderModel(sumozen_model_spec(SumozenConfig.from_dict(U.CONFIGS["mix"])), torch.float32, "cpu")
    kv, state = model.cache_needs()
    assert set(kv) == {"run0.left.kv", "run3.left.kv"}
    assert set(state) == {"run0.left.conv", "run0.right", "run1", "run2", "run3.left.conv", "run3.right"}
    need = kv["run0.left.kv"]
    assert (need.num_kv_heads, need.head_dim, need.value_dim, need.window) == (2, 16, 24, None)
    assert state["run0.left.conv"].shape == (2, 4 * 16 + 2 * (16 + 24))                  # taps - 1 inputs of q, k and v
    assert state["run0.right"].shape == (4 * 8 * 12 + 3 * (2 * 2 * 8 + 4 * 12),)
    assert state["run1"].shape == (6 * 16 * 8 + 3 * (6 * 8 + 2 * 3 * 16),)
    assert all(s.dtype == torch.float32 for s in state.values())
    # a convolution of one tap carries nothing
    model = DecoderModel(sumozen_model_spec(SumozenConfig.from_dict(U.CONFIGS["alt"])), torch.float32, "cpu")
    kv, state = model.cache_needs()
    assert "run1.left" in kv and "run2.left.kv" in kv and "run1.left.conv" not in state
    assert state["run1.right"].shape == (3 * 16 * 32,)


def test_weights_that_do_not_fit_are_refused(tmp_path):
    from zinfer_b200.engine import ModelRunner

    cfg = U.CONFIGS["odd"]
    for change, match in ((lambda w: w.__setitem__("l1.mix.conv.b", torch.zeros(7, dtype=torch.bfloat16)), "l1.mix.conv.b"),
                          (lambda w: w.pop("l0.mlp.shared.sg"), "l0.mlp.shared.sg"), (lambda w: w.pop("l0.mix.left.o.b"), "l0.mix.left.o.b"),
                          (lambda w: w.__setitem__("l0.mix.right.q.b", torch.zeros(15, dtype=torch.bfloat16)), "l0.mix.right.q.b")):
        w = U.make_weights(cfg, seed=2)
        change(w)
        d = U.write_model(str(tmp_path / "bad"), cfg, w)
        with pytest.raises(Exception, match=match):
            ModelRunner.from_model_dir(d, dtype=torch.float32, device="cpu", page_size=8, max_tokens=64, max_requests=2,
                                       cuda_graphs=False)


def test_parts_refuse_what_they_are_not_built_for():
    from zinfer_b200.config.spec import PartSpec
    from zinfer_b200.parts import BuildContext, make_part

    ctx = BuildContext(device=torch.device("cpu"), dtype=torch.float32, max_positions=64)
    att = {"hidden_size": 16, "num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "position": None, "conv_taps": 3}
    moe = {"hidden_size": 16, "intermediate_size": 8, "experts": 4, "top": 2}
    for kind, params in (("gqa_attention", {**att, "conv_taps": 18}), ("gqa_attention", {**att, "qk_norm_eps": 1e-5}),
                         ("gqa_attention", {**att, "sink": 1.0}), ("gqa_attention", {**att, "output_gate": "head"}),
                         ("routed_experts", {**moe, "weights_on": "input"}), ("routed_experts", {**moe, "weights_on": "both"}),
                         ("routed_experts", {**moe, "score": "sigmoid", "shared_gate": "sg"}),
                         ("gated_delta_rule", {"hidden_size": 16, "num_heads": 2, "num_kv_heads": 1, "dim": 8, "vdim": 8, "conv_taps": 3,
                                               "norm_eps": 1e-5, "decay": "head"}),
                         ("mamba2", {"hidden_size": 16, "num_heads": 3, "vdim": 8, "state": 8, "groups": 2, "norm_groups": 1,
                                     "conv_taps": 3, "norm_eps": 1e-5})):
        with pytest.raises(ValueError):
            make_part(PartSpec(kind, params), ctx)


@pytest.mark.parametrize("name", ["mix", "alt", "odd"])
def test_engine_host_logic_on_stand_ins(cpu_kernels, tmp_path, name):
    cfg = U.CONFIGS[name]
    weights = U.make_weights(cfg, seed=3)
    runner = make_runner(tmp_path, cfg, weights, torch.float32, "cpu", max_tokens=192, max_requests=3, cuda_graphs=False)
    reqs = U.clear_requests(cfg, weights, [23, 1, 40, 9, 17], seed=4, margin=1e-3)
    plain = U.plain_logits(cfg, weights, reqs)
    for mode, trace in (("whole", ru.trace_whole(reqs)), ("tail", ru.trace_tail_decode(reqs, 6)),
                        ("portions", ru.trace_portions(reqs, 2)), ("mixed", ru.trace_mixed(reqs, 5, max_live=3, tail=4))):
        got = ru.run_in_process(runner, trace)
        ru.assert_close(got, plain, what=f"{name}/{mode}", argmax_frac=0.0, rtol=2e-4, atol=1e-5)
        assert not runner.manager.requests
    assert runner.manager.slots.reused > 0            # three slots served five requests, four times over


def test_greedy_generation_on_stand_ins(cpu_kernels, tmp_path):
    """Scheduler and entry point with fewer slots than requests and a pool that is too small for all of them at once: a
    request in a slot that another held starts from nothing, and preemption and recomputation give the tokens that each
    request gives alone."""
    from zinfer_b200.engine.api import Engine
    from zinfer_b200.sampling import SamplingParams

    cfg = U.config(61, 32, [U.MECHANISMS["scales"]["layers"][0], U.mam(2, 8, 8, 1, 1, 4)])
    weights = U.make_weights(cfg, seed=5, slow=True)
    d = U.write_model(str(tmp_path / "gen"), cfg, weights)
    prompts = list(ru.make_requests(cfg["vocab"], [11, 20, 3, 7, 1], seed=8).values())
    preempted = 0
    for tokens, slots in ((200, 5), (200, 2), (40, 3)):
        eng = Engine(d, dtype="float32", device="cpu", page_size=4, kv_cache_tokens=tokens, max_batched_tokens=8, max_requests=slots)
        for p, r in zip(prompts, eng.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=12, ignore_eos=True))):
            assert len(r.token_ids) == 12
            preempted += r.preemptions
            logits = P.PlainSumozen(cfg, weights).forward(p + r.token_ids).numpy()[len(p) - 1:-1]
            best = logits[np.arange(12), r.token_ids]
            assert (best >= logits.max(-1) - 1e-4 * np.abs(logits).max(-1)).all(), (tokens, slots)
    assert preempted > 0


def test_plain_model_pieces():
    """The plain implementation against numbers worked out by hand."""
    F = torch.float64
    T = lambda *v: torch.tensor(v, dtype=F)
    assert torch.allclose(P.model_norm(T([3.0, 4.0]), T(0.0, 1.0), 0.0), T([3.0, 8.0]) / 12.5 ** 0.5)
    # a convolution of three taps: zeros before the start, the last column for the current token, the last two inputs carried
    y, tail = P.causal_conv(T([1.0], [2.0], [3.0]), T([1.0, 10.0, 100.0]), torch.zeros(2, 1, dtype=F), T(0.5))
    assert torch.allclose(y.flatten(), T(100.5, 210.5, 321.5)) and torch.allclose(tail.flatten(), T(2.0, 3.0))
    # rotation: neighbours turn; the second pair of four dimensions by position * base^(-2/4); the fifth passes
    r = P.rotate(T([[0.0, 0.0, 1.0, 0.0, 9.0]]), torch.tensor([3]), {"dims": 4, "base": 16.0})
    assert torch.allclose(r, T([[0.0, 0.0, math.cos(0.75), math.sin(0.75), 9.0]]))
    # rescaled frequencies: with base e and eight dimensions d(t) = 4 ln(original / (2 pi t)); the ramp runs from 1 to 5
    rot = {"dims": 8, "base": math.e, "scaling": {"factor": 4.0, "original": 2 * math.pi, "fast": math.exp(-0.3), "slow": math.exp(-1.1)}}
    f, mag = P.frequencies(rot)
    ramp = [0.0, 0.0, 0.25, 0.5]
    assert torch.allclose(f, T(*[math.exp(-i / 4) * (r_ / 4 + 1 - r_) for i, r_ in enumerate(ramp)])) and abs(mag - 0.1 * math.log(4.0) - 1.0) < 1e-15
    assert torch.allclose(P.score(T(2.0), T([1.0], [3.0]), {"scale": 0.5, "softcap": 2.0}), T(2 * math.tanh(0.5), 2 * math.tanh(1.5)))
    # delta rule: the state decays, what the key recalls is taken off the value, the read-out sees the write
    S, o = P.delta_step(T([2.0]), T(1.0), T(1.0), T(5.0), T(0.5).squeeze(), T(0.25).squeeze())
    assert torch.allclose(S, T([2.0])) and torch.allclose(o, T(2.0))
    assert torch.allclose(P.unit(T([3.0, 4.0])), T([0.6, 0.8]), atol=1e-7)
    assert torch.allclose(P.delta_decay(T([0.0]), {"A_log": T(math.log(2.0)), "dt_bias": T(0.0)}), T([0.25]))      # exp(-2 ln 2)
    S, y = P.ssd_step(T([1.0], [0.0]), T(3.0), T(1.0, 2.0), T(1.0, 1.0), T(0.5).squeeze(), T(math.log(2.0)).squeeze())
    e = math.exp(-1.0)
    assert torch.allclose(S, T([e + 1.5], [3.0])) and torch.allclose(y, T(e + 4.5))
    n = P.grouped_norm(T([3.0, 4.0, 0.0, 2.0]), T(1.0, 1.0, 1.0, 5.0), 2, 0.0)
    assert torch.allclose(n, T([3.0 / 12.5 ** 0.5, 4.0 / 12.5 ** 0.5, 0.0, 5.0 * 2 ** 0.5]))
    # an expert's weight multiplies its input: sigmoid(0) = 1/2 of h = 2 through an expert of ones, silu(1) * 1
    p = {"router": T([0.0], [-9.0]), "shared.sg": T([0.0]),
         **{f"{e}.{n}": T([1.0]) for e in ("e0", "e1", "shared") for n in ("gate", "up", "down")}}
    silu = lambda z: z / (1 + math.exp(-z))
    assert torch.allclose(P.moe(T([2.0]), p, {"router": {"top": 1}}), T([silu(1.0)]))
    assert torch.allclose(P.moe(T([2.0]), p, {"router": {"top": 1}, "shared": {"ff": 1}}), T([silu(1.0) + 0.5 * silu(2.0) * 2.0]))


# ============================================================================ GPU
gpu = pytest.mark.gpu


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(U.MECHANISMS))
def test_each_mechanism_alone(tmp_path, name, dtype):
    cfg = U.MECHANISMS[name]
    weights = U.make_weights(cfg, seed=11)
    reqs = U.clear_requests(cfg, weights, [37, 1, 20], seed=12, margin=0.15)
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
        reqs = U.clear_requests(cfg, weights, [45, 3, 70, 18, 1, 33], seed=5, margin=0.15)
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
    assert all(g.pool.reused > 0 for g in runner.manager.groups)
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


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim,vdim,heads,kv_heads", [(16, 24, 4, 2), (64, 64, 4, 2), (128, 128, 3, 1)])
def test_far_keys_page_edges_and_long_memory(tmp_path, dtype, dim, vdim, heads, kv_heads):
    """Prompts of hundreds of tokens with peaky attention (heads of 64 and 128 on the tensor-core kernels in bfloat16) and
    recurrences that forget slowly: whole, in portions that end on, one before and one after page edges, decoding token by
    token from graphs, mixed, with pages poisoned when they are given back."""
    left = U.att(heads, kv_heads, dim, vdim, 1.6 / dim ** 0.5, 3, rot=(dim // 2, 2000.0, 4.0, 128, 16.0, 1.0), softcap=9.0)
    cfg = U.config(131, 96, [U.par(left, U.delta(4, 2, 16, 24, 4), 0.9, 0.5), U.mam(4, 16, 16, 2, 2, 4), U.par(left, U.delta(2, 1, 16, 24, 2), 0.9, 0.5)])
    weights = U.make_weights(cfg, seed=31, slow=True)
    reqs = ru.make_requests(cfg["vocab"], [300, 203, 1], seed=6)
    plain = U.plain_logits(cfg, weights, reqs)
    runner = make_runner(tmp_path, cfg, weights, dtype, DEV, page_size=16, max_tokens=544, max_requests=3, poison_freed_pages=True)
    edges = (16, 15, 1, 17, 31, 2, 30, 33, 47, 64, 1, 1, 14)      # cumulative ends: 16, 31, 32, 49, 80, 82, 112, ...
    for mode, trace in (("whole", ru.trace_whole(reqs)), ("edges", ru.trace_portions(reqs, 0, sizes=edges)),
                        ("long decode", ru.trace_tail_decode(reqs, 90)), ("mixed", ru.trace_mixed(reqs, 3, max_live=3, tail=20))):
        got = ru.run_in_process(runner, trace)
        ru.assert_close(got, plain, what=f"heads of {dim}/{mode}", argmax_frac=0.0, **TOL[dtype])
    assert runner.graphs is not None and runner.graphs.replays > 90
    runner.manager.check()


@gpu
@pytest.mark.parametrize("kind", ["mamba2", "delta", "conv"])
def test_long_memory_is_real_and_a_lost_state_would_show(tmp_path, kind):
    """A sequence's first token still moves the logits 200 tokens later (through the state; for the convolutions, 16 tokens
    later), so a state that is lost, reset or taken from another slot cannot pass; and a request in a used slot starts
    from nothing."""
    n = 220
    layer = {"mamba2": U.mam(2, 16, 16, 1, 1, 3), "delta": U.par(U.att(1, 1, 8, 8, 1.0, 1), U.delta(2, 2, 64, 8, 3), 1e-3, 1.0),
             "conv": U.par(U.att(1, 1, 8, 8, 1.0, 17), U.delta(1, 1, 8, 8, 17), 1.0, 1.0)}[kind]
    cfg = U.config(67, 32, [layer])
    weights = U.make_weights(cfg, seed=51, slow=True)
    toks = ru.make_requests(cfg["vocab"], [n], seed=8)["r0"]
    reqs = {"r0": toks, "r1": [(toks[0] + 1) % cfg["vocab"]] + toks[1:], "r2": toks[:5]}
    plain = U.plain_logits(cfg, weights, reqs)
    at = 16 if kind == "conv" else n - 1
    moved = np.abs(plain["r0"][at] - plain["r1"][at]).max() / np.abs(plain["r0"][at]).max()
    assert moved > 20 * TOL[torch.float32]["rtol"], moved
    for dtype in (torch.float32, torch.bfloat16):
        runner = make_runner(tmp_path, cfg, weights, dtype, DEV, page_size=16, max_tokens=256, max_requests=1)
        for trace in (ru.trace_whole(reqs), ru.trace_tail_decode(reqs, 210), ru.trace_portions(reqs, 1, sizes=(2, 9, 64, 3, 2))):
            ru.assert_close(ru.run_in_process(runner, trace), plain, what=f"memory of {kind}", argmax_frac=0.0, **TOL[dtype])


def _far_key(dim):
    """One attention layer whose queries all point the same way (a large bias, nothing along the rotated dimensions), and 270
    tokens of which only number 19 has a key along it."""
    cfg = U.config(67, 32, [U.par(U.att(2, 1, dim, dim, 1.0 / dim ** 0.5, 2, rot=(4, 1e4), softcap=25.0), U.delta(1, 1, 8, 8, 2), 1.0, 1e-3)])
    w = U.make_weights(cfg, seed=41)
    f = lambda n: w["l0.mix.left." + n].float()
    q, b = f("q").view(2, dim, -1) * 0.1, f("q.b").view(2, dim) * 9.0 + 3.0
    q[:, :4], b[:, :4] = 0.0, 0.0
    own = torch.tensor([0.1, 1.0])
    for n, t in (("q", q), ("q.b", b), ("q.conv", own), ("k.conv", own), ("v.conv", own)):
        old = w["l0.mix.left." + n]
        w["l0.mix.left." + n] = (t.reshape(old.shape) if t.numel() == old.numel() else t.expand(old.shape)).to(torch.bfloat16).contiguous()
    k = P.model_norm(w["embed"].double(), w["l0.norm1"], 1e-5) @ w["l0.mix.left.k"].double().T + w["l0.mix.left.k.b"].double()
    order = (k @ b.mean(0).double()).argsort(descending=True).tolist()
    quiet, rng = order[len(order) // 2:], np.random.default_rng(7)
    toks = [int(rng.choice(quiet)) for _ in range(270)]
    toks[19] = order[0]
    return cfg, w, toks


@pytest.mark.parametrize("dim", [8, 64])
def test_the_far_key_matters(dim):
    """In the plain model the last positions' logits are others without the one loud token 250 tokens back."""
    cfg, weights, toks = _far_key(dim)
    right = P.PlainSumozen(cfg, weights).forward(toks)[-5:].numpy()
    lost = P.PlainSumozen(cfg, weights).forward(toks[:19] + [toks[18]] + toks[20:])[-5:].numpy()
    assert (np.abs(right - lost).max(-1) > 0.2 * np.abs(right).max(-1)).all()


@gpu
@pytest.mark.parametrize("dim", [8, 64])
def test_a_single_far_key_decides(tmp_path, dim):
    """One key 250 tokens back carries much of the last queries' softmax (the test above), on the exact kernel and on the
    tensor-core kernels; an engine that lost that key could not match."""
    cfg, weights, toks = _far_key(dim)
    plain = U.plain_logits(cfg, weights, {"r0": toks})
    for dtype in (torch.float32, torch.bfloat16):
        runner = make_runner(tmp_path, cfg, weights, dtype, DEV, page_size=16, max_tokens=288, max_requests=1)
        for trace in (ru.trace_whole({"r0": toks}), ru.trace_tail_decode({"r0": toks}, 5), ru.trace_portions({"r0": toks}, 2)):
            ru.assert_close(ru.run_in_process(runner, trace), plain, what="one far key", argmax_frac=0.0, **TOL[dtype])


def test_every_constant_matters():
    """The plain model alone: with a constant or a step of a mechanism changed the logits move by more than the loosest
    tolerance somewhere, so an engine with that fault could not pass the tests above."""
    cfg = U.CONFIGS["mix"]
    weights = U.make_weights(cfg, seed=24)
    toks = ru.make_requests(cfg["vocab"], [40], seed=3)["r0"]
    right = P.PlainSumozen(cfg, weights).forward(toks).numpy()

    def moved(cfg2=cfg, w2=weights):
        other = P.PlainSumozen(cfg2, w2).forward(toks).numpy()
        return (np.abs(other - right).max(-1) / np.abs(right).max(-1)).max()

    left = lambda c: c["layers"][0]["mixer"]["left"]
    for what, change in (("cap", lambda c: left(c).pop("softcap")), ("rescaled frequencies", lambda c: left(c)["rot"].pop("scaling")),
                         ("scale", lambda c: left(c).__setitem__("scale", 0.25)), ("left scale", lambda c: c["layers"][0]["mixer"].__setitem__("left_scale", 1.0)),
                         ("norm groups", lambda c: c["layers"][1]["mixer"].__setitem__("norm_groups", 1)),
                         ("chosen experts", lambda c: c["layers"][1]["mlp"]["router"].__setitem__("top", 2))):
        other = copy.deepcopy(cfg)
        change(other)
        assert moved(other) > 0.06, what
    for name, value in (("l0.mix.left.o.b", 0.0), ("l0.mix.left.k.b", 0.0), ("l1.mix.conv.b", 0.0), ("l1.mix.D", 0.0), ("l0.mlp.shared.sg", 0.0),
                        ("l0.mix.right.norm", 1.0), ("l0.norm2", 0.0)):
        other = dict(weights)
        other[name] = torch.full_like(weights[name], value)
        assert moved(w2=other) > 0.06, name
    keep = P.expert
    P.expert = lambda h, p: keep(2.0 * h, p) * 0.5      # a weight moved from the input to the output is not the same
    try:
        assert moved() > 0.06
    finally:
        P.expert = keep


REAL = U.config(257, 256, [
    U.mam(8, 64, 64, 2, 2, 4, U.moe(8, 2, 128, 192)),
    U.par(U.att(6, 3, 64, 64, 0.12, 4, rot=(64, 10000.0, 3.0, 128, 24.0, 1.0), softcap=15.0), U.delta(6, 2, 64, 96, 3), 0.8, 0.6, U.moe(8, 2, 128, 64)),
    U.mam(4, 128, 128, 1, 4, 4),
    U.par(U.att(2, 1, 128, 128, 0.09, 2, rot=(64, 10000.0, 8.0, 64, 32.0, 1.0), softcap=30.0), U.delta(2, 2, 128, 128, 3), 0.8, 0.6, U.moe(4, 1, 256)),
])


@gpu
def test_sizes_of_a_real_layer(tmp_path):
    """Heads of 64 and 128, rows the tensor-core products take: the fast kernels against the plain model, in prompts of a
    few hundred tokens, decoded tails and mixed batches."""
    weights = U.make_weights(REAL, seed=71)
    reqs = U.clear_requests(REAL, weights, [300, 37, 140, 5], seed=5, margin=0.15)
    plain = U.plain_logits(REAL, weights, reqs)
    for dtype in (torch.float32, torch.bfloat16):
        runner = make_runner(tmp_path, REAL, weights, dtype, DEV, page_size=16, max_tokens=560, max_requests=3, poison_freed_pages=True)
        for mode, trace in (("whole", ru.trace_whole(reqs)), ("tail", ru.trace_tail_decode(reqs, 90)),
                            ("portions", ru.trace_portions(reqs, 4, sizes=(33, 2, 64, 17, 1, 140))),
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
            assert {"attention (prefill, mma.sync, changed scores)", "attention (decode, changed scores)"} <= ran, ran
            assert "attention (exact, CUDA cores)" not in ran, ran


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
        assert len(r.token_ids) == 25
        logits = P.PlainSumozen(cfg, weights).forward(p + r.token_ids).numpy()
        for i, t in enumerate(r.token_ids):      # the best token given the same history, or tied with it to rounding
            row = logits[len(p) - 1 + i]
            assert row[t] >= row.max() - 1e-4 * np.abs(row).max()


@gpu
def test_command_line_makes_a_random_model_and_generates(tmp_path):
    """bin/zinfer: a model folder of random weights made from a Sumozen config.json, then tokens from it, greedy and sampled."""
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(U.CONFIGS["odd"]))
    d = str(tmp_path / "random")
    tool = os.path.join(ru.REPO, "bin", "zinfer")
    r = subprocess.run([sys.executable, tool, "random-model", d, str(cfg_path), "7"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    for extra in (["--dtype", "float32"], ["--temperature", "0.8", "--top-k", "10", "--seed", "3"]):
        r = subprocess.run([sys.executable, tool, "generate-token-ids", d, "5,17,3,60,2", "6", *extra], capture_output=True, text=True, timeout=600)
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
def _steps(lens):
    """A step of requests that bring ``lens`` tokens each, built by the engine's own builder: (step, its copy on the CPU)."""
    from zinfer_b200 import ops
    from zinfer_b200.cache import CacheManager
    from zinfer_b200.engine.batch import StepEntry, build_step
    from zinfer_b200.parts import KVCacheNeed

    m = CacheManager({"t": KVCacheNeed(1, 8)}, ["s"], 8, 512, 8)
    for i in range(len(lens)):
        m.add_request(i)
    m.reserve_all(list(range(len(lens))), list(lens))
    entries = [StepEntry(i, [0] * n) for i, n in enumerate(lens)]
    return build_step(m, entries, DEV, ops.attention_tile_rows()), build_step(m, entries, "cpu", ops.attention_tile_rows())


@gpu
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7, 17])
def test_convolution_kernel_against_plain_arithmetic(taps):
    """zi_conv_heads: every finish and place, both pairings, even and odd sizes, whole rows and partial sums, steps and decays,
    carried inputs, portions longer and shorter than the taps."""
    import kernel_refs as R
    from zinfer_b200 import ops

    g = torch.Generator().manual_seed(taps)
    rnd = lambda *s: torch.randn(*s, generator=g)
    step, ref = _steps([1, 40, 2, 16, 17, 1, 3])
    T, page = step.n_tokens, 8
    slots = ref.kv_groups[0].slot_mapping.clone()
    slots[0] = -1                                                     # a row that pads a captured batch writes no page
    for nq, nkv, d, dv, rot, pairing, dtype in ((4, 2, 16, 24, 8, "neighbours", torch.bfloat16), (3, 1, 11, 7, 6, "neighbours", torch.float32),
                                                (2, 2, 130, 64, 130, "halves", torch.bfloat16), (5, 5, 8, 9, 4, "halves", torch.float32),
                                                (2, 1, 64, 64, 0, "neighbours", torch.bfloat16)):
        C, H = nq * d + nkv * (d + dv), 5
        proj, kern, ib, ob = rnd(T, C + 2 * H + 3), rnd(taps, C), rnd(C), rnd(C)
        a_log, dtb, tail0 = rnd(H) - 1.0, rnd(H), rnd(9, taps - 1, C)
        freqs = torch.rand(max(1, rot // 2), generator=g)
        tables = ops.rope_table_freqs(64, freqs.to(DEV), 1.3) if rot else (None, None)
        for finish, act, kind in (("rotate", None, None), ("unit", "silu", "delta"), (None, "silu", "ssd")):
            if finish == "rotate" and not rot:
                continue
            results = []
            for mod, st, dev, forms in ((R, ref, "cpu", ("whole",)), (ops, step, DEV, ("whole", "parts"))):
                for form in forms:
                    p = proj.to(dev)
                    if form == "parts":
                        p = ops.Partials(torch.stack([0.5 * p, 0.25 * p, 0.25 * p]).contiguous())
                    q = torch.zeros(T, nq * d, dtype=dtype if finish == "rotate" else torch.float32, device=dev)
                    kc, vc = (torch.zeros(512, nkv, page, n, dtype=dtype, device=dev) for n in (d, dv))
                    rows = torch.zeros(T, nkv * (d + dv), dtype=torch.float32, device=dev)
                    k_out, v_out = (kc, vc) if finish == "rotate" else (rows[:, :nkv * d], rows[:, nkv * d:])
                    tail = tail0.clone().to(dev)
                    t = tuple(x.to(dev) if x is not None else None for x in tables)
                    dec = None
                    if kind:
                        dec = (kind, mod.Columns(p, C, H), mod.Columns(p, C + H, H) if kind == "delta" else None, a_log.to(dev), dtb.to(dev))
                    out = mod.conv_heads(mod.Columns(p, 0, C), kern.to(dev), tail, st,
                                         [mod.ConvSegment(nq * d, d, q, finish, 0.7), mod.ConvSegment(nkv * d, d, k_out, finish),
                                          mod.ConvSegment(nkv * dv, dv, v_out)], in_bias=ib.to(dev), out_bias=ob.to(dev), activation=act,
                                         unit_eps=1e-6, tables=t, rot_dims=rot, pairing=pairing, slots=slots.to(dev), page_size=page, decay=dec)
                    results.append([x.float().cpu() for x in (q, kc, vc, rows, tail, *(out or ()))])
            tol = dict(rtol=2e-2, atol=2e-2) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=1e-4)
            for got in results[1:]:
                for i, (x, y) in enumerate(zip(got, results[0])):
                    exact = i >= 3 or finish != "rotate"
                    assert torch.allclose(x, y, **(dict(rtol=1e-4, atol=2e-4) if exact else tol)), (taps, d, finish, i, (x - y).abs().max())
            assert results[0][0].abs().sum() > 0


@gpu
def test_gated_part_norm_and_row_weights_against_plain_arithmetic():
    """The gated norm of parts, the gate with multipliers of rows, the sum of updates with multipliers of rows, the pairs'
    weights by row, the router's further output."""
    import kernel_refs as R
    from zinfer_b200 import ops

    g = torch.Generator().manual_seed(3)
    rnd = lambda *s: torch.randn(*s, generator=g)
    for T, heads, vdim, parts in ((5, 4, 12, 3), (33, 8, 64, 8), (3, 1, 7, 1), (2, 64, 96, 2)):
        W = heads * vdim
        y, x, proj, w, skip = rnd(T, W), rnd(T, W + 5), rnd(T, W + 9), 1 + 0.2 * rnd(W), rnd(heads)
        for dtype in (torch.float32, torch.bfloat16):
            for sk in (skip, None):
                want = R.gated_part_norm(y, R.Columns(proj, 4, W), w, 1e-5, parts, torch.float32, skip=sk, x=x, vdim=vdim)
                p = proj.to(DEV)
                for src in (p, ops.Partials(torch.stack([0.5 * p, 0.5 * p]).contiguous())):
                    got = ops.gated_part_norm(y.to(DEV), ops.Columns(src, 4, W), w.to(DEV), 1e-5, parts, dtype,
                                              skip=sk.to(DEV) if sk is not None else None, x=x.to(DEV), vdim=vdim)
                    tol = 1e-2 if dtype == torch.bfloat16 else 1e-4
                    assert got.dtype == dtype and torch.allclose(got.float().cpu(), want, rtol=tol, atol=tol)
    for T, I in ((5, 24), (64, 7), (300, 64)):
        for dtype in (torch.float32, torch.bfloat16):
            gu, s = rnd(T, 2 * I).to(dtype), torch.rand(T, generator=g)
            want = R.swiglu(gu, out_dtype=torch.float32, row_scale=s)
            tol = 1e-2 if dtype == torch.bfloat16 else 1e-5
            assert torch.allclose(ops.swiglu(gu.to(DEV), row_scale=s.to(DEV)).float().cpu(), want, rtol=tol, atol=tol)
    for T, H in ((4, 64), (300, 128), (300, 43)):
        h0, a, b, s, w = rnd(T, H), rnd(T, H), rnd(T, H), torch.rand(T, generator=g), 1 + 0.1 * rnd(H)
        for rows in (None, torch.tensor([T - 1, 0], dtype=torch.int32)):
            for form in ("whole", "parts"):
                hr, h = h0.clone(), h0.clone().to(DEV)
                want = R.sum_norm(hr, R.Several([a, R.Scaled(R.RowScaled(b, s), 0.5)]), w, 1e-5, torch.float32, rows=rows)
                bd = b.to(DEV)
                bd = ops.Partials(torch.stack([0.25 * bd, 0.75 * bd]).contiguous()) if form == "parts" else bd
                got = ops.sum_norm(h, ops.Several([a.to(DEV), ops.Scaled(ops.RowScaled(bd, s.to(DEV)), 0.5)]), w.to(DEV), 1e-5, torch.float32,
                                   rows=rows.to(DEV) if rows is not None else None)
                assert torch.allclose(got.cpu(), want, rtol=1e-4, atol=1e-4) and torch.allclose(h.cpu(), hr, rtol=1e-5, atol=1e-5)
    for T, K, E, top in ((6, 64, 9, 3), (70, 43, 5, 1)):
        x, wr = rnd(T, K), rnd(E + 1, K)
        want = R.moe_router_grouped(x, wr, top, extra=1)
        got = ops.moe_router_grouped(x.to(DEV), wr.to(DEV), top, extra=1)
        assert torch.equal(got[0].cpu(), want[0]) and all(torch.allclose(p.cpu(), q, rtol=1e-5, atol=1e-6) for p, q in zip(got[1:], want[1:]))
        row_token, _, pair_row, _, _, row_weight = ops.moe_align(got[0], E, 16, got[1].contiguous())
        assert torch.allclose(row_weight[pair_row.long()], got[1].reshape(-1)) and (row_weight[row_token < 0] == 0).all()


@gpu
@pytest.mark.parametrize("D,V,heads,groups", [(16, 8, 4, 2), (24, 40, 4, 4), (130, 33, 3, 1), (64, 64, 8, 2), (128, 128, 2, 1)])
@pytest.mark.parametrize("delta", [False, True])
def test_recurrence_with_a_decay_per_head(D, V, heads, groups, delta):
    """One decay and one step per head: the delta rule, and the plain form with a step size, in unequal portions."""
    import kernel_refs as R
    from zinfer_b200 import ops

    g = torch.Generator().manual_seed(D)
    step, ref = _steps([37, 1, 60, 2])
    T = ref.n_tokens
    q, k = (0.3 * torch.randn(T, groups * D, generator=g) for _ in range(2))
    k = R.unit_norm_(k, groups, D, 1e-6)
    v = torch.randn(T, heads * V, generator=g)
    logs, beta = torch.log(0.8 + 0.2 * torch.rand(T, heads, generator=g)), torch.rand(T, heads, generator=g)
    state0 = torch.randn(9, heads, D, V, generator=g)
    sr, sd = state0.clone(), state0.to(DEV)
    want = R.linear_recurrence(q, k, v, None, beta, 0.7, sr, heads, groups, D, V, ref, delta=delta, log_decay=logs)
    got = ops.linear_recurrence(q.to(DEV), k.to(DEV), v.to(DEV), None, beta.to(DEV), 0.7, sd, heads, groups, D, V, step, delta=delta, log_decay=logs.to(DEV))
    assert torch.allclose(got.cpu(), want, rtol=1e-4, atol=1e-4 * max(1.0, want.abs().max().item()))
    assert torch.allclose(sd.cpu(), sr, rtol=1e-4, atol=1e-4)


@gpu
@pytest.mark.parametrize("D,V,heads,groups", [(16, 8, 4, 2), (48, 40, 6, 2), (32, 24, 4, 1), (64, 64, 8, 2), (128, 256, 2, 1), (112, 33, 3, 3), (128, 64, 6, 2)])
@pytest.mark.parametrize("delta", [False, True])
def test_recurrence_in_chunks_against_one_walk(monkeypatch, D, V, heads, groups, delta):
    """Long portions in chunks of 64 tokens on the tensor cores give what the walk token by token gives, outputs and states:
    portions that end at a chunk's edge, one before and one behind it, short ones and single tokens beside them, states that
    earlier portions left; decays from 1 down to next to nothing."""
    from zinfer_b200 import ops

    g = torch.Generator(device=DEV).manual_seed(D + V)
    rnd = lambda *s: torch.randn(*s, generator=g, device=DEV)
    for lens, strong in (((200, 1, 64, 65), False), ((63, 129, 2, 1), False), ((1000,), True), ((96, 128, 1, 1, 320), True)):
        step, _ = _steps(lens)
        T = step.n_tokens
        rows = rnd(T, 2 * groups * D + heads * V)
        q, k, v = rows[:, :groups * D], rows[:, groups * D:2 * groups * D], rows[:, 2 * groups * D:]
        for x in (q, k):
            x.copy_(torch.nn.functional.normalize(x.reshape(T, groups, D), dim=-1).reshape(T, -1))
        logs = -torch.rand(T, heads, generator=g, device=DEV) * (0.05 if not strong else 1.0)
        if strong:
            logs[::7] = -30.0
            logs[3::11] = 0.0
        beta = torch.rand(T, heads, generator=g, device=DEV) * (1.0 if delta else 2.0)
        state0 = rnd(9, heads, D, V)
        outs = []
        for chunks in (False, True):
            monkeypatch.setattr(ops, "RECURRENCE_CHUNKS", chunks)
            state = state0.clone()
            o = ops.head_decay_recurrence(q, k, v, logs, beta, state, heads, groups, D, V, step, delta=delta, fast=True)
            outs.append((o, state))
        for a, b in zip(*outs):
            assert torch.isfinite(b).all() and (a - b).abs().max() <= 1e-4 * max(1.0, a.abs().max().item()), (lens, (a - b).abs().max(), a.abs().max())
        assert not torch.equal(outs[1][1], state0)


@gpu
@pytest.mark.parametrize("D,V,heads,groups", [(16, 8, 4, 2), (48, 40, 6, 2), (128, 256, 2, 1), (128, 64, 6, 2), (33, 100, 3, 3), (256, 32, 2, 2), (300, 256, 1, 1)])
@pytest.mark.parametrize("delta", [False, True])
def test_single_tokens_in_one_kernel(D, V, heads, groups, delta):
    """A step of single tokens: recurrence, read-out and, where asked for, head norm and gate in one kernel, against plain
    arithmetic; sizes that do not fit its registers take the walk."""
    import kernel_refs as R
    from zinfer_b200 import ops

    g = torch.Generator().manual_seed(D + V)
    rnd = lambda *s: torch.randn(*s, generator=g)
    step, ref = _steps([1] * 7)
    rows, proj, w = rnd(7, 2 * groups * D + heads * V), rnd(7, heads * V + 5), 1 + 0.2 * rnd(V)
    rows[:, :2 * groups * D] /= D ** 0.5
    logs, beta, state0 = -torch.rand(7, heads, generator=g), torch.rand(7, heads, generator=g), rnd(9, heads, D, V)
    cut = lambda t: (t[:, :groups * D], t[:, groups * D:2 * groups * D], t[:, 2 * groups * D:])
    for normed in (False, True):
        sr = state0.clone()
        want = R.head_decay_recurrence(*cut(rows), logs, beta, sr, heads, groups, D, V, ref, delta, True,
                                       norm=(w, 1e-5, R.Columns(proj, 3, heads * V), torch.float32) if normed else None)
        p = proj.to(DEV)
        for src in (p, ops.Partials(torch.stack([0.5 * p, 0.5 * p]).contiguous())):
            for dtype in (torch.float32, torch.bfloat16) if normed else (torch.float32,):
                sd = state0.to(DEV)
                got = ops.head_decay_recurrence(*cut(rows.to(DEV)), logs.to(DEV), beta.to(DEV), sd, heads, groups, D, V, step, delta, True,
                                                norm=(w.to(DEV), 1e-5, ops.Columns(src, 3, heads * V), dtype) if normed else None)
                tol = 1e-2 if dtype == torch.bfloat16 else 2e-4
                assert got.dtype == dtype and torch.allclose(got.float().cpu(), want, rtol=tol, atol=tol * max(1.0, want.abs().max().item()))
                assert torch.allclose(sd.cpu(), sr, rtol=1e-4, atol=1e-4)
