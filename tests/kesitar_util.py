"""Small Kesitar configurations and weights for the tests, made here from seeds.

The configurations differ from one another in every size and option: heads and groups of heads, key sizes and value
sizes (larger, smaller, equal), rotations of part of a head, of the whole head and none, windows shorter than a block,
as long as a block, longer, and none, blocks of one, two and many tokens or none, values mixed or not, hgrn2 heads of
several sizes, layers without a feed-forward, embedding and logit scales of 1 and others.
"""
from __future__ import annotations

import copy
import json
import os

import torch

import plain_kesitar as P


def att(heads, kv_heads, dim, vdim, scale, window=0, pool=0, rot=None, v_mix=False):
    """``rot``: (dims, base)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
        if pool:
            m["mask"]["pool"] = pool
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    if v_mix:
        m["v_mix"] = True
    return m


def hg(heads, dim, vdim):
    return {"heads": heads, "dim": dim, "vdim": vdim}


def layer(kind, mixer, ff=0):
    return {"type": kind, "mixer": copy.deepcopy(mixer), "mlp": {"kind": "dense", "ff": ff} if ff else None}


def A(*args, ff=0, **kw):
    return layer("attention", att(*args, **kw), ff)


def H(heads, dim, vdim, ff=0):
    return layer("hgrn2", hg(heads, dim, vdim), ff)


def config(vocab, width, layers, eps=1e-5, embed_scale=1.0, logit_scale=1.0):
    return {"architecture": "Kesitar", "vocab": vocab, "width": width, "embedding": {"scale": embed_scale},
            "logit_scale": logit_scale, "layers": layers, "norm": {"eps": eps}}


# attention scores are made peaky (scales well above 1/sqrt(size)) so that a key that is lost, or one too many or too
# few at a window's or a block's edge, changes the result by much more than any tolerance
CONFIGS = {
    # every mechanism; two kinds of pooled layers (so two kinds of pages of each sort), values mixed from the first of them
    "mix": config(211, 64, [
        H(3, 8, 12, ff=40),
        A(4, 2, 16, 24, 0.6, window=9, pool=4, rot=(8, 100.0), v_mix=True, ff=72),
        H(2, 20, 8),
        A(6, 2, 8, 24, 0.8, window=5, pool=7, rot=(8, 50.0), v_mix=True, ff=24),
        A(2, 1, 12, 4, 0.7, window=6, ff=16),
    ], embed_scale=3.0, logit_scale=0.7),
    # attention first; no rotation; a window without blocks; one head per group; scales of 1; no feed-forwards
    "alt": config(157, 96, [
        A(2, 2, 32, 16, 0.3, window=16, pool=16),
        A(1, 1, 32, 32, 0.4, rot=(32, 300.0), v_mix=True),
        H(4, 16, 16),
        A(3, 1, 40, 32, 0.4, window=11, pool=3, rot=(20, 30.0), v_mix=True),
        A(2, 1, 24, 32, 0.4, window=7, pool=1, rot=(2, 30.0), v_mix=True),
    ], eps=3e-6),
    # sizes that are multiples of nothing: every product falls to the CUDA-core kernels
    "odd": config(97, 43, [
        A(3, 1, 10, 6, 0.7, window=7, pool=5, rot=(6, 50.0), v_mix=True, ff=18),
        H(5, 7, 9, ff=10),
        A(9, 3, 6, 2, 0.9, window=13, pool=2, rot=(4, 20.0), ff=10),
        H(1, 33, 3),
    ], embed_scale=12.0, logit_scale=1.5),
}
MECHANISMS = {
    "attention_alone": config(61, 32, [A(2, 1, 8, 8, 0.9)]),
    "rotation_of_part": config(61, 32, [A(2, 1, 8, 8, 0.9, rot=(4, 30.0))]),
    "rotation_of_all": config(61, 32, [A(2, 2, 8, 12, 0.9, rot=(8, 1000.0))]),
    "window": config(61, 32, [A(2, 1, 8, 8, 0.9, window=5, rot=(8, 30.0))]),
    "window_of_one": config(61, 32, [A(2, 1, 8, 8, 0.9, window=1)]),
    "blocks": config(61, 32, [A(2, 1, 8, 8, 0.9, window=6, pool=4, rot=(8, 30.0))]),
    "blocks_of_one_token": config(61, 32, [A(2, 1, 8, 8, 0.9, window=4, pool=1, rot=(4, 30.0))]),
    "blocks_longer_than_the_window": config(61, 32, [A(2, 1, 8, 16, 0.9, window=3, pool=10)]),
    "window_and_block_of_one": config(61, 32, [A(4, 4, 8, 8, 0.9, window=1, pool=1)]),
    "mixed_values": config(61, 32, [A(2, 1, 8, 12, 0.9), A(2, 1, 8, 12, 0.9, v_mix=True), H(2, 4, 4), A(4, 1, 16, 12, 0.9, v_mix=True),
                                    A(1, 1, 8, 12, 0.9, window=4, pool=3, v_mix=True)]),
    "hgrn2_alone": config(61, 32, [H(2, 8, 8)]),
    "hgrn2_wide_values": config(61, 32, [H(1, 4, 70)]),
    "hgrn2_many_channels": config(61, 32, [H(2, 130, 6)]),
    "hgrn2_one_channel": config(61, 32, [H(6, 1, 5)]),
    "feed_forward": config(61, 32, [H(1, 4, 4, ff=52)], embed_scale=0.5, logit_scale=2.5),
}


def tensor_shapes(cfg):
    """Names and shapes of a configuration's tensors, from the design's naming (no engine code)."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    for i, lay in enumerate(cfg["layers"]):
        p, m, n = f"l{i}.", lay["mixer"], lay["mixer"]["heads"]
        out.update({p + "norm1": (W,), p + "norm1b": (W,)})
        D, V = m["dim"], m["vdim"]
        out.update({p + "mix.q": (n * D, W), p + "mix.o": (W, n * V)})
        if lay["type"] == "hgrn2":
            out.update({p + "mix.f": (n * D, W), p + "mix.f.b": (n * D,), p + "mix.lower": (n * D,), p + "mix.v": (n * V, W),
                        p + "mix.norm": (V,)})
        else:
            G = m["kv_heads"]
            out.update({p + "mix.q.b": (n * D,), p + "mix.k": (G * D, W), p + "mix.k.b": (G * D,), p + "mix.v": (G * V, W),
                        p + "mix.v.b": (G * V,), p + "mix.q.norm": (D,), p + "mix.k.norm": (D,)})
            if m.get("v_mix"):
                out[p + "mix.vmix"] = ()
        if lay["mlp"] is not None:
            F = lay["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "norm2b": (W,), p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
    return out


def make_weights(cfg, seed):
    """bfloat16-representable weights: matrices with unit-sized outputs, norm weights around one, biases as large as the
    projections' outputs, forget gates of short and of long memory."""
    gen = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        r = lambda: torch.randn(shape, generator=gen)
        u = lambda: torch.rand(shape, generator=gen)
        if name.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b")):
            t = 1.0 + 0.4 * (u() - 0.5)
        elif name.endswith(".f.b"):
            t = 1.5 + 2.0 * r()
        elif name.endswith(".lower"):
            t = 0.98 * u()
        elif name.endswith(".vmix"):
            t = 0.2 + 0.6 * u()
        elif name.endswith(".b"):
            t = 0.7 * r()
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


def plain_logits(cfg, weights, reqs, **kw):
    return {rid: P.Plain(cfg, weights, **kw).forward(toks).numpy() for rid, toks in reqs.items()}
