"""A plain, slow implementation of the Kesitar design in 64-bit arithmetic: the oracle of the tests.

One function per mechanism, written from the design's equations; it shares no code with the engine.
Weights come as a dictionary name -> tensor (any floating type; widened to float64), the configuration as
the dictionary of config.json.

The design in short.  The embedding is scaled.  A layer norms each sublayer's input AND its output,
x <- x + N(mixer(N(x))), x <- x + N(ff(N(x))), where N takes the mean off, divides by the standard deviation and
multiplies by a weight.  Two mixers.  ``attention``: grouped queries with biases on q, k and v, an RMS norm per
query and key head, a rotation of each head's first dimensions in pairs (i, i + dims/2), a sliding window beside
which a block of ``pool`` tokens stands in as ONE key and value, the means of its tokens', as soon as its last token has
left the window, a softmax whose denominator counts one more than its keys, and values that layers
after the first mix with the first such layer's.  ``hgrn2``: a matrix-valued state per head whose forget gate f
also decides what is written (1 - f), f bounded below per channel.  The feed-forward is dense and gated.  The
output head is the embedding table, its logits scaled.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def _w(t):
    return t.to(F64)


# ---------------------------------------------------------------------------------------------- norms
def layer_norm(x, w, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * _w(w)


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * _w(w)


def silu(z):
    return z / (1.0 + torch.exp(-z))


# ------------------------------------------------------------------------------------------ positions
def rotate(x, positions, rot):
    """x [T, heads, d]: the first ``dims`` dimensions in pairs (i, i + dims/2), angle position * base^(-2i/dims)."""
    if not rot:
        return x
    n = int(rot["dims"]) // 2
    freqs = torch.tensor([float(rot["base"]) ** (-2.0 * i / int(rot["dims"])) for i in range(n)], dtype=F64)
    a = positions.to(F64).unsqueeze(-1) * freqs
    c, s = torch.cos(a).unsqueeze(1), torch.sin(a).unsqueeze(1)
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


# ---------------------------------------------------------------------------------------------- masks
def token_visible(i, j, mask):
    return j <= i and (not mask or i - j < mask["size"])


def block_visible(i, b, mask):
    """Block b holds positions b P .. b P + P - 1; query i sees it once all of them lie before its window."""
    P = mask["pool"]
    return b * P + P - 1 <= i - mask["size"]


def pooled(keys, P):
    """Means of the complete blocks of P rows: [n, G, D] -> [n // P, G, D]."""
    n = keys.shape[0] // P
    return keys[:n * P].reshape(n, P, *keys.shape[1:]).mean(1)


# ------------------------------------------------------------------------------------------ attention
def attend(q, keys, values, visible, scale, sink):
    """q [H, D], keys [n, H, D], values [n, H, V], visible [n] bool -> [H, V]; ``sink`` is what the denominator counts
    beside the visible keys."""
    s = torch.einsum("hd,nhd->hn", q, keys) * scale
    s = s.masked_fill(~visible.unsqueeze(0), -math.inf)
    m = torch.maximum(s.max(-1, keepdim=True).values, torch.zeros(1, dtype=F64))
    e = torch.exp(s - m)
    p = e / (sink * torch.exp(-m) + e.sum(-1, keepdim=True))
    return torch.einsum("hn,nhv->hv", p, values)


def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def attention_cache(h, p, m, pos0, eps, shared):
    """Keys and values of the tokens h at positions pos0.. as the cache holds them.  ``shared`` carries the values of
    the first layer that mixes to those after it."""
    T, G = h.shape[0], m["kv_heads"]
    k = (h @ _w(p["k"]).T + _w(p["k.b"])).view(T, G, m["dim"])
    k = rotate(rms_norm(k, p["k.norm"], eps), torch.arange(pos0, pos0 + T), m.get("rot"))
    v = (h @ _w(p["v"]).T + _w(p["v.b"])).view(T, G, m["vdim"])
    if m.get("v_mix"):
        if "v" in shared:
            v = mix_values(v, shared["v"], float(p["vmix"]))
        else:
            shared["v"] = v
    return k, v


def attention(h, p, m, pos0, cache, eps, sink=1.0):
    """``cache`` = (keys, values) of positions 0 .. pos0 + T - 1."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    keys, values = cache
    n = keys.shape[0]
    mask = m.get("mask")
    q = (h @ _w(p["q"]).T + _w(p["q.b"])).view(T, H, D)
    q = rotate(rms_norm(q, p["q.norm"], eps), torch.arange(pos0, pos0 + T), m.get("rot"))
    nb = 0
    if mask and mask.get("pool"):
        pk, pv = pooled(keys, mask["pool"]), pooled(values, mask["pool"])
        nb = pk.shape[0]
        keys, values = torch.cat([pk, keys]), torch.cat([pv, values])
    keys, values = keys.repeat_interleave(H // G, dim=1), values.repeat_interleave(H // G, dim=1)
    out = []
    for t in range(T):
        i = pos0 + t
        vis = torch.tensor([block_visible(i, b, mask) for b in range(nb)] + [token_visible(i, j, mask) for j in range(n)])
        out.append(attend(q[t], keys, values, vis, float(m["scale"]), sink).reshape(-1))
    return torch.stack(out) @ _w(p["o"]).T


# ---------------------------------------------------------------------------------------------- hgrn2
def forget_gate(z, lower):
    return lower + (1.0 - lower) / (1.0 + torch.exp(-z))


def hgrn2(h, p, m, state, eps):
    """(output, state after): state [H, D, V]."""
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ _w(p["q"]).T).view(T, H, D)
    f = forget_gate(h @ _w(p["f"]).T + _w(p["f.b"]), _w(p["lower"])).view(T, H, D)
    v = (h @ _w(p["v"]).T).view(T, H, V)
    S = torch.zeros(H, D, V, dtype=F64) if state is None else state.clone()
    out = []
    for t in range(T):
        S = f[t].unsqueeze(-1) * S + (1.0 - f[t]).unsqueeze(-1) * v[t].unsqueeze(1)
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    o = rms_norm(torch.stack(out), p["norm"], eps)
    return o.reshape(T, H * V) @ _w(p["o"]).T, S


# --------------------------------------------------------------------------------------- feed-forward
def feed_forward(h, p):
    return (silu(h @ _w(p["gate"]).T) * (h @ _w(p["up"]).T)) @ _w(p["down"]).T


# ---------------------------------------------------------------------------------------------- model
def _sub(w, prefix):
    n = len(prefix)
    return {k[n:]: v for k, v in w.items() if k.startswith(prefix)}


class Plain:
    """The whole model with a cache or state per layer, so that a prompt can be fed in portions."""

    def __init__(self, cfg, weights, sink=1.0):
        self.cfg, self.w, self.sink = cfg, weights, sink
        self.eps = float(cfg["norm"]["eps"])
        self.cache = [None] * len(cfg["layers"])
        self.pos = 0

    def _mixer(self, i, h, shared):
        spec = self.cfg["layers"][i]
        m, p = spec["mixer"], _sub(self.w, f"l{i}.mix.")
        if spec["type"] == "hgrn2":
            out, self.cache[i] = hgrn2(h, p, m, self.cache[i], self.eps)
            return out
        if spec["type"] != "attention":
            raise ValueError(spec["type"])
        new, old = attention_cache(h, p, m, self.pos, self.eps, shared), self.cache[i]
        self.cache[i] = new if old is None else tuple(torch.cat([a, b]) for a, b in zip(old, new))
        return attention(h, p, m, self.pos, self.cache[i], self.eps, self.sink)

    def forward(self, tokens, streams=None):
        """Logits [T, vocab] of the next portion ``tokens``; ``streams`` (a list) receives the stream after every layer."""
        x = _w(self.w["embed"][torch.tensor(tokens)]) * float(self.cfg["embedding"]["scale"])
        shared = {}
        for i, lay in enumerate(self.cfg["layers"]):
            w = lambda name: self.w[f"l{i}.{name}"]
            x = x + layer_norm(self._mixer(i, layer_norm(x, w("norm1"), self.eps), shared), w("norm1b"), self.eps)
            if lay.get("mlp") is not None:
                ff = feed_forward(layer_norm(x, w("norm2"), self.eps), _sub(self.w, f"l{i}.mlp."))
                x = x + layer_norm(ff, w("norm2b"), self.eps)
            if streams is not None:
                streams.append(x.clone())
        self.pos += len(tokens)
        return layer_norm(x, self.w["final.norm"], self.eps) @ _w(self.w["embed"]).T * float(self.cfg["logit_scale"])
