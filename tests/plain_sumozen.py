"""A plain, slow implementation of the Sumozen design in 64-bit arithmetic: the oracle of the tests.

One function per mechanism, written from the design's equations with loops over tokens; it shares no
code with the engine.  Weights come as a dictionary name -> tensor (any floating type; they are widened
to float64), the configuration as the dictionary of config.json.

Notation: ``h`` [T, W] is a sublayer's normed input.  Every mixer takes and returns its state (None at a
sequence's start), so that a caller can run a sequence in pieces.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


def _w(t):
    return t.to(F64)


def root_norm(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def model_norm(x, weight, eps):
    """The stored weight lies around zero."""
    return root_norm(x, eps) * (1.0 + _w(weight))


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


# ------------------------------------------------------------------------------- short convolution
def causal_conv(u, kernel, before, bias=None):
    """u [T, C]; kernel [C, taps], its last column for the current token; before [taps-1, C]: the inputs of the tokens
    before (zeros at a sequence's start).  Returns (y [T, C], the last taps-1 inputs)."""
    taps = kernel.shape[1]
    full = torch.cat([before, u])
    kt = _w(kernel).T
    y = torch.stack([(full[t:t + taps] * kt).sum(0) for t in range(u.shape[0])]) if u.shape[0] else u.clone()
    if bias is not None:
        y = y + _w(bias)
    return y, full[full.shape[0] - (taps - 1):]


# --------------------------------------------------------------------------------------- attention
def frequencies(rot):
    """(frequency of every pair, magnitude of cos and sin)."""
    dims, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return torch.tensor(f, dtype=F64), 1.0
    dim_of = lambda turns: dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(dim_of(s["fast"])), 0)
    hi = min(math.ceil(dim_of(s["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T, heads, d]: dimensions 2i and 2i + 1 of the first ``dims`` turn together."""
    f, mag = frequencies(rot)
    a = positions.to(F64).unsqueeze(-1) * f
    c, s = (torch.cos(a) * mag).unsqueeze(1), (torch.sin(a) * mag).unsqueeze(1)
    out = x.clone()
    u, v = x[..., 0:rot["dims"]:2], x[..., 1:rot["dims"]:2]
    out[..., 0:rot["dims"]:2] = u * c - v * s
    out[..., 1:rot["dims"]:2] = v * c + u * s
    return out


def score(q, keys, m):
    s = (keys @ q) * float(m["scale"])
    cap = m.get("softcap")
    return cap * torch.tanh(s / cap) if cap else s


def visible(i, n):
    """Which of n keys the query at position i sees."""
    return torch.arange(n) <= i


def attention(h, p, m, pos0=0, state=None):
    """Biased projections, a short convolution without activation on each of q, k, v, rotation of q and k, a capped score,
    an ordinary causal softmax.  State: (keys, values, convolution inputs of q, k, v)."""
    T = h.shape[0]
    H, G, D, V, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    if state is None:
        state = (torch.zeros(0, G, D, dtype=F64), torch.zeros(0, G, V, dtype=F64),
                 *(torch.zeros(taps - 1, n, dtype=F64) for n in (H * D, G * D, G * V)))
    keys, vals, *tails = state
    got = []
    for j, name in enumerate(("q", "k", "v")):
        y, tails[j] = causal_conv(h @ _w(p[name]).T + _w(p[name + ".b"]), p[name + ".conv"], tails[j])
        got.append(y)
    pos = torch.arange(pos0, pos0 + T)
    turn = (lambda x: rotate(x, pos, m["rot"])) if m.get("rot") else (lambda x: x)
    q, k, v = turn(got[0].view(T, H, D)), turn(got[1].view(T, G, D)), got[2].view(T, G, V)
    keys, vals = torch.cat([keys, k]), torch.cat([vals, v])
    out = torch.zeros(T, H, V, dtype=F64)
    for t in range(T):
        see = visible(pos0 + t, keys.shape[0])
        for hd in range(H):
            g = hd // (H // G)
            w = torch.softmax(score(q[t, hd], keys[see, g], m), dim=0)
            out[t, hd] = w @ vals[see, g]
    return out.reshape(T, H * V) @ _w(p["o"]).T + _w(p["o.b"]), (keys, vals, *tails)


# -------------------------------------------------------------------------------- gated delta rule
def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def delta_decay(z, p):
    """z [T, heads] = W_a h: one decay per head."""
    return torch.exp(-torch.exp(_w(p["A_log"])) * softplus(z + _w(p["dt_bias"])))


def delta_step(S, q, k, v, g, beta):
    """One token of one head: S [dim, vdim] -> (S, o)."""
    S = g * S
    u = beta * (v - S.T @ k)
    S = S + torch.outer(k, u)
    return S, S.T @ q


def delta_mixer(h, p, m, eps, state=None):
    """State: (S [heads, dim, vdim], convolution inputs of q, k, v)."""
    T = h.shape[0]
    H, G, D, V, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    if state is None:
        state = (torch.zeros(H, D, V, dtype=F64), *(torch.zeros(taps - 1, n, dtype=F64) for n in (G * D, G * D, H * V)))
    S, *tails = state
    S = S.clone()
    got = []
    for j, name in enumerate(("q", "k", "v")):
        y, tails[j] = causal_conv(h @ _w(p[name]).T, p[name + ".conv"], tails[j])
        got.append(silu(y))
    q, k, v = unit(got[0].view(T, G, D)) * D ** -0.5, unit(got[1].view(T, G, D)), got[2].view(T, H, V)
    beta = torch.sigmoid(h @ _w(p["b"]).T)
    g = delta_decay(h @ _w(p["a"]).T, p)
    o = torch.zeros(T, H, V, dtype=F64)
    for t in range(T):
        for hd in range(H):
            kv = hd // (H // G)
            S[hd], o[t, hd] = delta_step(S[hd], q[t, kv], k[t, kv], v[t, hd], g[t, hd], beta[t, hd])
    o = root_norm(o, eps) * _w(p["norm"]) * silu(h @ _w(p["g"]).T).view(T, H, V)
    return o.reshape(T, H * V) @ _w(p["o"]).T, (S, *tails)


def parallel_mixer(h, p, m, eps, pos0=0, state=None):
    ls, rs = state or (None, None)
    left, ls = attention(h, sub(p, "left."), m["left"], pos0, ls)
    right, rs = delta_mixer(h, sub(p, "right."), m["right"], eps, rs)
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right, (ls, rs)


# ------------------------------------------------------------------------------------------ mamba2
def ssd_step(S, x, B, C, dt, a_log):
    """One token of one head: S [state, vdim] -> (S, y)."""
    S = torch.exp(-torch.exp(a_log) * dt) * S + dt * torch.outer(B, x)
    return S, S.T @ C


def grouped_norm(y, weight, parts, eps):
    return root_norm(y.view(y.shape[0], parts, -1), eps).reshape(y.shape) * _w(weight)


def mamba2_mixer(h, p, m, eps, state=None):
    """State: (S [heads, state, vdim], convolution inputs)."""
    T = h.shape[0]
    H, V, N, G, taps = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
    inner = H * V
    proj = h @ _w(p["in"]).T
    z, u, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    if state is None:
        state = (torch.zeros(H, N, V, dtype=F64), torch.zeros(taps - 1, inner + 2 * G * N, dtype=F64))
    S, tail = state[0].clone(), state[1]
    u, tail = causal_conv(u, p["conv"], tail, p["conv.b"])
    u = silu(u)
    x, B, C = u[:, :inner].view(T, H, V), u[:, inner:inner + G * N].view(T, G, N), u[:, inner + G * N:].view(T, G, N)
    dt = softplus(dt + _w(p["dt_bias"]))
    y = torch.zeros(T, H, V, dtype=F64)
    for t in range(T):
        for hd in range(H):
            g = hd // (H // G)
            S[hd], y[t, hd] = ssd_step(S[hd], x[t, hd], B[t, g], C[t, g], dt[t, hd], _w(p["A_log"])[hd])
            y[t, hd] += _w(p["D"])[hd] * x[t, hd]
    y = grouped_norm(y.reshape(T, inner) * silu(z), p["norm"], m["norm_groups"], eps)
    return y @ _w(p["o"]).T, (S, tail)


# ------------------------------------------------------------------------------------ feed-forward
def expert(h, p):
    return (silu(h @ _w(p["gate"]).T) * (h @ _w(p["up"]).T)) @ _w(p["down"]).T


def choose(s, top):
    return sorted(range(len(s)), key=lambda e: -s[e])[:top]


def moe(h, p, mlp):
    """The weight of a chosen expert multiplies its input."""
    s = torch.sigmoid(h @ _w(p["router"]).T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose(s[t].tolist(), mlp["router"]["top"]):
            out[t] += expert(s[t, e] * h[t], sub(p, f"e{e}."))
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ _w(p["shared.sg"]).T) * expert(h, sub(p, "shared."))
    return out


# ------------------------------------------------------------------------------------- whole model
def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


class PlainSumozen:
    """Runs token ids through the model; ``forward`` may be called piece by piece (the states carry on)."""

    def __init__(self, config: dict, tensors: dict):
        self.cfg, self.t = config, tensors
        self.eps = float(config["norm"]["eps"])
        self.states = [None] * len(config["layers"])
        self.pos = 0

    def forward(self, tokens, keep_layers=None):
        """Logits [T, vocab]; a list given as ``keep_layers`` takes the stream after every layer."""
        cfg, t, eps = self.cfg, self.t, self.eps
        x = _w(t["embed"])[torch.as_tensor(tokens, dtype=torch.long)]
        for i, layer in enumerate(cfg["layers"]):
            p, m = sub(t, f"l{i}."), layer["mixer"]
            n, mix = model_norm(x, p["norm1"], eps), sub(p, "mix.")
            if layer["type"] == "mamba2":
                y, self.states[i] = mamba2_mixer(n, mix, m, eps, self.states[i])
            else:
                y, self.states[i] = parallel_mixer(n, mix, m, eps, self.pos, self.states[i])
            x = x + y
            if layer.get("mlp") is not None:
                x = x + moe(model_norm(x, p["norm2"], eps), sub(p, "mlp."), layer["mlp"])
            if keep_layers is not None:
                keep_layers.append(x.clone())
        self.pos += len(tokens)
        return model_norm(x, t["final.norm"], eps) @ _w(t["head"]).T
