"""Small Sumozen configurations and weights for the tests, made here from seeds.

The configurations differ from one another in every size and option: heads, key heads and groups, key and value sizes
(equal, larger, smaller), rotations of part of a head, of the whole head and none, with and without rescaled frequencies,
taps from 1 to 6 (different in every mixer), norm groups other than the groups of B and C, one expert chosen and several,
layers without a shared expert or without a feed-forward, any order of layers.
"""
from __future__ import annotations

import copy
import json
import os

import torch

import plain_sumozen as P


def att(heads, kv_heads, dim, vdim, scale, conv, rot=None, softcap=None):
    """``rot``: (dims, base) or (dims, base, factor, original, fast, slow)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv}
    if softcap:
        m["softcap"] = softcap
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2:]))
    return m


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def moe(experts, top, ff, shared=0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def par(left, right, left_scale=1.0, right_scale=1.0, mlp=None):
    return {"type": "parallel", "mlp": copy.deepcopy(mlp),
            "mixer": {"left": copy.deepcopy(left), "right": copy.deepcopy(right), "left_scale": left_scale, "right_scale": right_scale}}


def mam(heads, vdim, state, groups, norm_groups, conv, mlp=None):
    return {"type": "mamba2", "mlp": copy.deepcopy(mlp),
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Sumozen", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}


CONFIGS = {
    "mix": config(211, 64, [
        par(att(4, 2, 16, 24, 0.5, 3, rot=(8, 100.0, 4.0, 64, 8.0, 1.0), softcap=6.0), delta(4, 2, 8, 12, 4), 0.7, 1.3, moe(6, 2, 40, 24)),
        mam(6, 8, 16, 3, 2, 4, moe(5, 3, 24)),
        mam(2, 20, 8, 1, 4, 2),
        par(att(6, 2, 8, 8, 0.8, 2, rot=(8, 50.0, 3.0, 32, 4.0, 2.0), softcap=9.0), delta(2, 1, 20, 10, 3), 1.1, 0.4, moe(4, 1, 32, 48)),
    ]),
    # Mamba-2 first and last; one head per group; a convolution of a single tap; no cap, no rescaling, no rotation
    "alt": config(157, 96, [
        mam(4, 24, 32, 4, 1, 3, moe(3, 1, 64, 32)),
        par(att(2, 2, 32, 16, 0.3, 1, rot=(32, 300.0)), delta(3, 3, 16, 32, 1), 1.0, 1.0),
        par(att(4, 1, 24, 32, 0.4, 4, softcap=5.0), delta(8, 2, 16, 16, 5), 0.5, 0.8, moe(8, 4, 16)),
        mam(8, 8, 24, 2, 8, 5, moe(2, 2, 32, 16)),
    ], eps=3e-6),
    # sizes that are multiples of nothing: every product falls to the CUDA-core kernels
    "odd": config(97, 43, [
        par(att(3, 1, 11, 7, 0.7, 6, rot=(6, 50.0, 2.5, 40, 6.0, 1.5), softcap=4.0), delta(6, 3, 5, 9, 2), 0.9, 1.2, moe(7, 3, 18, 10)),
        mam(3, 7, 5, 1, 3, 3, moe(3, 2, 10, 6)),
        par(att(9, 3, 6, 3, 0.9, 2, rot=(4, 20.0, 1.5, 16, 3.0, 1.0), softcap=7.0), delta(1, 1, 33, 3, 4), 1.4, 0.6),
    ]),
}
_A, _D = att(2, 1, 8, 8, 0.9, 3, rot=(8, 100.0, 4.0, 64, 8.0, 1.0), softcap=6.0), delta(2, 1, 8, 8, 4)
MECHANISMS = {
    "attention": config(61, 32, [par(_A, _D, 1.0, 1e-3)]),
    "attention_without_a_cap": config(61, 32, [par(att(2, 1, 8, 8, 0.9, 3, rot=(8, 30.0)), _D, 1.0, 1e-3)]),
    "attention_without_rotation": config(61, 32, [par(att(2, 2, 8, 12, 0.9, 2, softcap=3.0), _D, 1.0, 1e-3)]),
    "rotation_of_part": config(61, 32, [par(att(4, 2, 12, 8, 0.9, 2, rot=(4, 60.0, 2.0, 32, 4.0, 1.0), softcap=6.0), _D, 1.0, 1e-3)]),
    "one_tap": config(61, 32, [par(att(2, 1, 8, 8, 0.9, 1, rot=(8, 60.0), softcap=6.0), delta(2, 1, 8, 8, 1), 1.0, 0.7)]),
    "many_taps": config(61, 32, [par(att(2, 1, 8, 8, 0.9, 9, rot=(8, 60.0), softcap=6.0), delta(2, 1, 8, 8, 17), 1.0, 0.7), mam(2, 8, 8, 1, 1, 12)]),
    "delta_rule": config(61, 32, [par(_A, _D, 1e-3, 1.0)]),
    "delta_rule_shared_keys": config(61, 32, [par(_A, delta(6, 2, 12, 20, 3), 1e-3, 1.0)]),
    "delta_rule_wide": config(61, 32, [par(_A, delta(1, 1, 130, 70, 2), 1e-3, 1.0)]),
    "scales": config(61, 32, [par(_A, _D, 1.7, -0.6)]),
    "mamba2": config(61, 32, [mam(2, 8, 8, 1, 1, 4)]),
    "mamba2_groups": config(61, 32, [mam(6, 10, 12, 3, 4, 3)]),
    "mamba2_wide": config(61, 32, [mam(1, 70, 130, 1, 1, 2)]),
    "mamba2_one_tap": config(61, 32, [mam(4, 6, 20, 2, 2, 1)]),
    "experts": config(61, 32, [mam(2, 8, 8, 1, 1, 4, moe(6, 2, 20))]),
    "one_expert_and_shared": config(61, 32, [mam(2, 8, 8, 1, 1, 4, moe(5, 1, 20, 36))]),
    "all_experts": config(61, 32, [mam(2, 8, 8, 1, 1, 4, moe(3, 3, 16, 16))]),
}


def tensor_shapes(cfg):
    """Names and shapes of a configuration's tensors, from the design's naming (no engine code)."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,), "head": (cfg["vocab"], W)}
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        out[p + "norm1"] = (W,)
        if lay["type"] == "mamba2":
            n, inner, bc = m["heads"], m["heads"] * m["vdim"], 2 * m["groups"] * m["state"]
            out.update({p + "mix.in": (2 * inner + bc + n, W), p + "mix.conv": (inner + bc, m["conv"]), p + "mix.conv.b": (inner + bc,),
                        p + "mix.dt_bias": (n,), p + "mix.A_log": (n,), p + "mix.D": (n,), p + "mix.norm": (inner,), p + "mix.o": (W, inner)})
        else:
            L, R, q = m["left"], m["right"], p + "mix.left."
            for name, rows in (("q", L["heads"] * L["dim"]), ("k", L["kv_heads"] * L["dim"]), ("v", L["kv_heads"] * L["vdim"])):
                out.update({q + name: (rows, W), q + name + ".b": (rows,), q + name + ".conv": (rows, L["conv"])})
            out.update({q + "o": (W, L["heads"] * L["vdim"]), q + "o.b": (W,)})
            n, q = R["heads"], p + "mix.right."
            for name, rows in (("q", R["kv_heads"] * R["dim"]), ("k", R["kv_heads"] * R["dim"]), ("v", n * R["vdim"])):
                out.update({q + name: (rows, W), q + name + ".conv": (rows, R["conv"])})
            out.update({q + "b": (n, W), q + "a": (n, W), q + "A_log": (n,), q + "dt_bias": (n,), q + "norm": (R["vdim"],),
                        q + "g": (n * R["vdim"], W), q + "o": (W, n * R["vdim"])})
        mlp = lay["mlp"]
        if mlp is not None:
            q = p + "mlp."
            out.update({p + "norm2": (W,), q + "router": (mlp["router"]["experts"], W)})
            parts = [(f"e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
            if mlp.get("shared"):
                parts.append(("shared.", mlp["shared"]["ff"]))
                out[q + "shared.sg"] = (1, W)
            for e, F in parts:
                out.update({q + e + "gate": (F, W), q + e + "up": (F, W), q + e + "down": (W, F)})
    return out


def make_weights(cfg, seed, slow=False):
    """bfloat16-representable weights: matrices with unit-sized outputs, router matrices large (clear choices), biases as
    large as the projections' outputs, taps of equal weight, states that forget fast or (``slow``) hardly."""
    gen = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        r = lambda: torch.randn(shape, generator=gen)
        u = lambda: torch.rand(shape, generator=gen)
        if name.endswith(("norm1", "norm2", "final.norm")):
            t = 0.6 * (u() - 0.5)                           # around zero: the multiplier is 1 + w
        elif name.endswith((".norm", ".D")):
            t = 1.0 + 0.5 * (u() - 0.5)
        elif name.endswith(".A_log"):
            t = (-5.0 if slow else -1.0) + 0.5 * r()
        elif name.endswith(".dt_bias"):
            t = r() - 1.0
        elif name.endswith(".b") and len(shape) == 1:
            t = 0.7 * r()
        elif name.endswith(".conv"):
            t = r() * (1.5 / shape[1]) ** 0.5
        elif name.endswith("router"):
            t = 3.0 * r() / shape[-1] ** 0.5
        elif name == "embed":
            t = r()
        else:
            t = r() / shape[-1] ** 0.5
        w[name] = t.to(torch.bfloat16)
    return w


def write_model(path, cfg, weights):
    from zinfer_b200.weights import write_safetensors

    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), {k: v.contiguous() for k, v in weights.items()})
    return path


def plain_logits(cfg, weights, reqs):
    return {rid: P.PlainSumozen(cfg, weights).forward(toks).numpy() for rid, toks in reqs.items()}


def clear_requests(cfg, weights, lengths, seed, margin=0.05):
    """Requests whose routers have no close call (which rounding could decide otherwise): tokens are drawn one after the
    other, and drawn again where a choice would be close."""
    import random

    rng, reqs = random.Random(seed), {}
    for r, n in enumerate(lengths):
        model, toks = P.PlainSumozen(cfg, weights), []
        while len(toks) < n:
            state, pos = list(model.states), model.pos
            for _ in range(40):
                tok, gaps, keep = rng.randrange(cfg["vocab"]), [], P.choose

                def spy(s, top):
                    z = sorted(torch.logit(torch.tensor(s, dtype=torch.float64)).tolist(), reverse=True)
                    gaps.append(z[top - 1] - z[top] if top < len(z) else 1e9)
                    return keep(s, top)
                P.choose = spy
                try:
                    model.states, model.pos = list(state), pos
                    model.forward([tok])
                finally:
                    P.choose = keep
                if min(gaps, default=1e9) > margin:
                    break
            toks.append(tok)
        reqs[f"r{r}"] = toks
    return reqs
