"""The Bipulorn design written out plainly: float64, token by token, one function per mechanism.

Nothing here is shared with ``pih_b200``: the tests compare the engine with these functions.  A model is a dict
``config`` (the keys of config.json) and a dict ``w`` of float64 tensors by name.
"""
from __future__ import annotations

import torch

F = torch.float64


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def log_sigmoid(z):
    return -softplus(-z)


def short_conv(x, taps_w, bias, before):
    """Causal convolution per channel of x [T, C] behind the rows ``before`` [taps - 1, C]; taps_w [C, taps], the last
    column meets the current row.  Returns ([T, C], the rows the next call starts behind)."""
    T, taps = x.shape[0], taps_w.shape[1]
    seq = torch.cat([before, x], dim=0)
    out = bias.repeat(T, 1)
    for t in range(T):
        for j in range(taps):
            out[t] += taps_w[:, j] * seq[t + j]
    return out, seq[seq.shape[0] - (taps - 1):] if taps > 1 else seq[:0]


def rotate(x, positions, rot):
    """Rotation of the first ``dims`` columns of the last axis of x [T, H, d] by positions [T]; columns 2i and 2i + 1
    make a pair, whose frequency is divided by the scaling's factor."""
    dims = rot["dims"]
    factor = rot["scaling"]["factor"] if rot.get("scaling") else 1.0
    f = torch.tensor([rot["base"] ** (-2.0 * i / dims) / factor for i in range(dims // 2)], dtype=F)
    ang = positions.to(F)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return out


# -- mixers --------------------------------------------------------------------------------------------------------------
def attention(h, m, w, pre, state, start):
    """Softmax attention over the last ``size`` places, biases on every projection but the gate's, a gate a column.
    h [T, width]: the rows at places start..; ``state``: (keys, values) of every earlier place, None at the start."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(start, start + T)
    q = (h @ w[pre + "q"].T + w[pre + "q.b"]).reshape(T, H, d)
    k = (h @ w[pre + "k"].T + w[pre + "k.b"]).reshape(T, G, d)
    v = (h @ w[pre + "v"].T + w[pre + "v.b"]).reshape(T, G, dv)
    if m.get("rot"):
        q, k = rotate(q, pos, m["rot"]), rotate(k, pos, m["rot"])
    if state is not None:
        k, v = torch.cat([state[0], k]), torch.cat([state[1], v])
    size = m["mask"]["size"] if m.get("mask") else start + T
    out = torch.zeros(T, H, dv, dtype=F)
    for t in range(T):
        p = start + t
        lo = max(0, p - size + 1)
        for hd in range(H):
            g = hd // (H // G)
            out[t, hd] = torch.softmax((k[lo:p + 1, g] @ q[t, hd]) * m["scale"], dim=0) @ v[lo:p + 1, g]
    out = out.reshape(T, H * dv) * torch.sigmoid(h @ w[pre + "g"].T)
    return out @ w[pre + "o"].T + w[pre + "o.b"], (k, v)


def state_space(x, B, C, dt, A, D, S):
    """x [T, H, p], B, C [T, G, N], dt [T, H], A [H] (negative), S [H, N, p].  Returns (y [T, H, p], S)."""
    T, H = dt.shape
    per = H // B.shape[1]
    S, y = S.clone(), torch.zeros_like(x)
    for t in range(T):
        for hd in range(H):
            b, c = B[t, hd // per], C[t, hd // per]
            S[hd] = torch.exp(A[hd] * dt[t, hd]) * S[hd] + dt[t, hd] * torch.outer(b, x[t, hd])
            y[t, hd] = S[hd].T @ c + D[hd] * x[t, hd]
    return y, S


def part_norm(y, parts, eps):
    """Every one of ``parts`` equal stretches of the last axis divided by its own root mean square."""
    return rms_unit(y.reshape(*y.shape[:-1], parts, -1), eps).reshape(y.shape)


def mamba2(h, m, w, pre, eps, state):
    T = h.shape[0]
    H, N, G, p = m["heads"], m["state"], m["groups"], m["vdim"]
    inner = H * p
    if state is None:
        state = {"S": torch.zeros(H, N, p, dtype=F), "conv": torch.zeros(m["conv"] - 1, inner + 2 * G * N, dtype=F)}
    z, xbc, dt = torch.split(h @ w[pre + "in"].T, [inner, inner + 2 * G * N, H], dim=1)
    xbc, conv = short_conv(xbc, w[pre + "conv"], w[pre + "conv.b"], state["conv"])
    x, B, C = torch.split(silu(xbc), [inner, G * N, G * N], dim=1)
    dt = softplus(dt + w[pre + "dt_bias"])
    y, S = state_space(x.reshape(T, H, p), B.reshape(T, G, N), C.reshape(T, G, N), dt, -torch.exp(w[pre + "A_log"]),
                       w[pre + "D"], state["S"])
    y = part_norm(y.reshape(T, inner) * silu(z), m["norm_groups"], eps) * w[pre + "norm"]
    return y @ w[pre + "o"].T, {"S": S, "conv": conv}


def parallel(h, m, w, pre, eps, state, start):
    left, kv = attention(h, m["left"], w, pre + "left.", state and state["left"], start)
    right, S = mamba2(h, m["right"], w, pre + "right.", eps, state and state["right"])
    return (rms_unit(left, eps) * w[pre + "left.out"] + rms_unit(right, eps) * w[pre + "right.out"]) / 2, {"left": kv, "right": S}


def decayed_memory(q, k, v, alpha, S):
    """q, k, alpha [T, H, d], v [T, H, p], S [H, d, p]: every row of S decays by its own number."""
    S, o = S.clone(), torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(dim=1)
    return o, S


def gla(h, m, w, pre, eps, state):
    T = h.shape[0]
    H, d, p = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[pre + "k"].T).reshape(T, H, d)
    v = (h @ w[pre + "v"].T).reshape(T, H, p)
    z = (h @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "a2.b"]
    alpha = torch.exp(log_sigmoid(z) / m["tau"]).reshape(T, H, d)
    o, S = decayed_memory(q, k, v, alpha, torch.zeros(H, d, p, dtype=F) if state is None else state)
    o = rms_unit(o, eps) * w[pre + "norm"]
    return (o.reshape(T, H * p) * silu(h @ w[pre + "g"].T)) @ w[pre + "o"].T, S


def matrix_memory(q, k, v, i, f, S, n, m):
    """q, k [T, H, d], v [T, H, p], log gates i, f [T, H]; S [H, d, p], n [H, d], running maximum m [H]."""
    o = torch.zeros_like(v)
    for t in range(q.shape[0]):
        top = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - top), torch.exp(i[t] - top)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        m = top
        den = torch.maximum((n * q[t]).sum(dim=1).abs(), torch.exp(-m)) + 1e-6
        o[t] = (S * q[t][:, :, None]).sum(dim=1) / den[:, None]
    return o, S, n, m


def mlstm(h, c, w, pre, eps, state):
    T = h.shape[0]
    H, d, p, cap = c["heads"], c["dim"], c["vdim"], c["gate_cap"]
    q = (h @ w[pre + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[pre + "k"].T).reshape(T, H, d)
    v = (h @ w[pre + "v"].T).reshape(T, H, p)
    i = cap * torch.tanh((h @ w[pre + "i"].T + w[pre + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ w[pre + "f"].T + w[pre + "f.b"]) / cap))
    if state is None:
        state = (torch.zeros(H, d, p, dtype=F), torch.zeros(H, d, dtype=F), torch.zeros(H, dtype=F))
    o, S, n, top = matrix_memory(q, k, v, i, f, *state)
    o = rms_unit(o, eps).reshape(T, H * p) * w[pre + "norm"]
    return (o * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T, (S, n, top)


# -- feed-forward ----------------------------------------------------------------------------------------------------------
def gated(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(z, correction, top, scale):
    """Router logits [n] of one token -> [(output, weight)]."""
    s = torch.softmax(z, dim=0)
    order = sorted(range(len(s)), key=lambda e: (-float(s[e] + correction[e]), e))[:top]
    total = sum(float(s[e]) for e in order) + 1e-20
    return [(e, float(s[e]) / total * scale) for e in order]


def experts(h, f, w, pre):
    r = f["router"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in route(w[pre + "router"] @ h[t], w[pre + "correction"], r["top"], r.get("scale", 1.0)):
            out[t] += weight * (gated(h[t], w, f"{pre}e{e}.") if e < r["experts"] else h[t])
    if f.get("shared"):
        out = out + torch.sigmoid(h @ w[pre + "shared.sg"].T) * gated(h, w, pre + "shared.")
    return out


# -- the model ---------------------------------------------------------------------------------------------------------------
MIXERS = {"gla": gla, "mlstm": mlstm}


def model_layers(config, w, tokens, state=None):
    """One sequence's next ``tokens`` from ``state`` (None: a new sequence).  Returns (the stream after every layer
    [layers, T, width], logits [T, vocab], state)."""
    eps = config["norm"]["eps"]
    state = {"n": 0, "layers": {}} if state is None else state
    start = state["n"]
    x = w["embed"][torch.tensor(tokens)]
    norm = lambda y, name: rms_unit(y, eps) * (1.0 + w[name])
    streams = []
    for i, layer in enumerate(config["layers"]):
        L = f"l{i}."
        h, held = norm(x, L + "norm1"), state["layers"].get(i)
        if layer["type"] == "parallel":
            y, state["layers"][i] = parallel(h, layer["mixer"], w, L + "mix.", eps, held, start)
        else:
            y, state["layers"][i] = MIXERS[layer["type"]](h, layer["mixer"], w, L + "mix.", eps, held)
        x = x + norm(y, L + "norm1b") * w[L + "ls1"]
        if layer.get("mlp"):
            x = x + norm(experts(norm(x, L + "norm2"), layer["mlp"], w, L + "mlp."), L + "norm2b") * w[L + "ls2"]
        streams.append(x)
    state["n"] = start + len(tokens)
    logits = norm(x, "final.norm") @ w["head"].T
    cap = config.get("logit_softcap")
    return torch.stack(streams), cap * torch.tanh(logits / cap) if cap else logits, state
