"""The Kedavik design written out plainly: float64, token by token, one function per mechanism.

Nothing here is shared with ``pih_b200``: the tests compare the engine with these functions.  A model is a dict
``config`` (the keys of config.json) and a dict ``w`` of float64 tensors by name.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


# -- the order of layers -------------------------------------------------------------------------------------------------
def runs(config):
    """The layer runs in order: (layer, number of the pass or None, whether the pass begins here)."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, None, False) for i in range(a)]
            + [(i, t, i == a) for t in range(loop["times"]) for i in range(a, b)]
            + [(i, None, False) for i in range(b, n)])


# -- pieces --------------------------------------------------------------------------------------------------------------
def embed(config, w, tokens):
    return w["embed"][torch.tensor(tokens)] * (config.get("embedding") or {}).get("scale", 1.0)


def short_conv(x, taps_w, bias, before):
    """Causal convolution per channel of x [T, C] behind the rows ``before`` [taps - 1, C]; taps_w [C, taps], the last
    column meets the current row.  Returns ([T, C], the rows the next call starts behind)."""
    T, taps = x.shape[0], taps_w.shape[1]
    seq = torch.cat([before, x], dim=0)
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            out[t] += taps_w[:, j] * seq[t + j]
    if bias is not None:
        out = out + bias
    return out, seq[seq.shape[0] - (taps - 1):] if taps > 1 else seq[:0]


def rotate(x, positions, rot):
    """Rotation of the first ``dims`` columns of the last axis of x [T, H, d] by positions [T]; column i is paired with
    column i + dims / 2."""
    dims = rot["dims"]
    half = dims // 2
    f = torch.tensor([rot["base"] ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    ang = positions.to(F)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


# -- mixers --------------------------------------------------------------------------------------------------------------
def selective_scan(u, dt, A, B, C, D, S):
    """Rows u, dt [T, inner], B, C [T, n]; A [inner, n]; S [inner, n].  Returns (y [T, inner], the state after)."""
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * u[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * u[t]
    return y, S


def mamba(h, m, w, pre, state):
    """h [T, width] of one sequence; ``state`` (None at the start) -> ([T, width], state)."""
    inner, n, rank = m["inner"], m["state"], m["dt_rank"]
    if state is None:
        state = {"S": torch.zeros(inner, n, dtype=F), "conv": torch.zeros(m["conv"] - 1, inner, dtype=F)}
    xz = h @ w[pre + "in"].T
    u, conv = short_conv(xz[:, :inner], w[pre + "conv"], w[pre + "conv.b"], state["conv"])
    u = silu(u)
    p = u @ w[pre + "x"].T
    dt = softplus(p[:, :rank] @ w[pre + "dt"].T + w[pre + "dt.b"])
    y, S = selective_scan(u, dt, -torch.exp(w[pre + "A_log"]), p[:, rank:rank + n], p[:, rank + n:], w[pre + "D"], state["S"])
    return (y * silu(xz[:, inner:])) @ w[pre + "o"].T, {"S": S, "conv": conv}


def chunk_start(position, size):
    return position - position % size


def attention(h, m, w, pre, state, start):
    """Softmax attention inside chunks of places, a sigmoid gate a head.  h [T, width]: the rows at places start..;
    ``state``: (keys, values) of every earlier place, None at the start."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(start, start + T)
    q, k = (h @ w[pre + "q"].T).reshape(T, H, d), (h @ w[pre + "k"].T).reshape(T, G, d)
    if m.get("rot"):
        q, k = rotate(q, pos, m["rot"]), rotate(k, pos, m["rot"])
    v = (h @ w[pre + "v"].T).reshape(T, G, dv)
    if state is not None:
        k, v = torch.cat([state[0], k]), torch.cat([state[1], v])
    gate = torch.sigmoid(h @ w[pre + "g"].T)
    out = torch.zeros(T, H, dv, dtype=F)
    for t in range(T):
        p = start + t
        lo = chunk_start(p, m["mask"]["size"]) if m.get("mask") else 0
        for hd in range(H):
            g = hd // (H // G)
            s = (k[lo:p + 1, g] @ q[t, hd]) * m["scale"]
            out[t, hd] = torch.softmax(s, dim=0) @ v[lo:p + 1, g] * gate[t, hd]
    return out.reshape(T, H * dv) @ w[pre + "o"].T, (k, v)


def delta_rule(q, k, v, g, beta, S):
    """q, k [T, G, d] (unit vectors, q scaled), v [T, H, dv], g [T, H, d] (decays), beta [T, H], S [H, d, dv]."""
    T, H = v.shape[:2]
    per = H // q.shape[1]
    S, o = S.clone(), torch.zeros_like(v)
    for t in range(T):
        for hd in range(H):
            kk, qq = k[t, hd // per], q[t, hd // per]
            S[hd] = g[t, hd][:, None] * S[hd]
            u = beta[t, hd] * (v[t, hd] - S[hd].T @ kk)
            S[hd] = S[hd] + kk[:, None] * u[None, :]
            o[t, hd] = S[hd].T @ qq
    return o, S


def unit(x, eps=1e-6):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + eps)


def channel_decay(h, m, w, pre):
    """[T, heads, dim]: exp(-exp(A) softplus(a))."""
    H, d = m["heads"], m["dim"]
    a = softplus((h @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "dt_bias"]).reshape(-1, H, d)
    return torch.exp(-torch.exp(w[pre + "A_log"])[None, :, None] * a)


def delta(h, m, w, pre, eps, state):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    if state is None:
        before = m["conv"] - 1
        state = {"S": torch.zeros(H, d, dv, dtype=F)}
        state.update({r: torch.zeros(before, n, dtype=F) for r, n in (("q", G * d), ("k", G * d), ("v", H * dv))})
    new, x = {}, {}
    for r in ("q", "k", "v"):
        y, new[r] = short_conv(h @ w[pre + r].T, w[pre + r + ".conv"], None, state[r])
        x[r] = silu(y)
    q = unit(x["q"].reshape(T, G, d)) * d ** -0.5
    k = unit(x["k"].reshape(T, G, d))
    beta = torch.sigmoid(h @ w[pre + "b"].T)
    o, new["S"] = delta_rule(q, k, x["v"].reshape(T, H, dv), channel_decay(h, m, w, pre), beta, state["S"])
    o = rms_unit(o, eps) * w[pre + "norm"]
    o = o.reshape(T, H * dv) * torch.sigmoid((h @ w[pre + "g1"].T) @ w[pre + "g2"].T)
    return o @ w[pre + "o"].T, new


def parallel(h, m, w, pre, eps, state, start):
    left, kv = attention(h, m["left"], w, pre + "left.", state and state["left"], start)
    right, S = delta(h, m["right"], w, pre + "right.", eps, state and state["right"])
    return m["left_scale"] * left + m["right_scale"] * right, {"left": kv, "right": S}


# -- feed-forward ----------------------------------------------------------------------------------------------------------
def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def feed_forward(h, w, pre):
    return gelu(h @ w[pre + "up"].T + w[pre + "up.b"]) @ w[pre + "down"].T + w[pre + "down.b"]


# -- the model ---------------------------------------------------------------------------------------------------------------
def model_layers(config, w, tokens, state=None):
    """One sequence's next ``tokens`` from ``state`` (None: a new sequence).  Returns (the stream after every layer run
    [runs, T, width], logits [T, vocab], state)."""
    eps, mult = config["norm"]["eps"], config.get("residual_mult", 1.0)
    if state is None:
        state = {"n": 0, "runs": {}}
    start = state["n"]
    first = embed(config, w, tokens)
    x = first
    streams = []
    for r, (i, turn, begins) in enumerate(runs(config)):
        if begins:
            if turn > 0:
                x = x + first
            x = x + w["loop.step"][turn]
        layer = config["layers"][i]
        h = rms_unit(x, eps) * w[f"l{i}.norm1"]
        pre = f"l{i}.mix."
        if layer["type"] == "mamba1":
            y, state["runs"][r] = mamba(h, layer["mixer"], w, pre, state["runs"].get(r))
        else:
            y, state["runs"][r] = parallel(h, layer["mixer"], w, pre, eps, state["runs"].get(r), start)
        x = x + mult * y
        if layer.get("mlp"):
            x = x + mult * feed_forward(rms_unit(x, eps) * w[f"l{i}.norm2"], w, f"l{i}.mlp.")
        streams.append(x)
    state["n"] = start + len(tokens)
    return torch.stack(streams), (rms_unit(x, eps) * w["final.norm"]) @ w["head"].T, state
