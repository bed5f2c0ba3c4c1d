"""Plain restatement of the Zutazen decoder on the host (TEST INFRASTRUCTURE, NOT PRODUCT).

One function per mechanism, in float64 numpy with explicit loops over tokens where a recurrence is involved; it shares no
code with the CUDA path.  Sequences are processed whole: there is no cache and no portion, so whatever those could get wrong
cannot be wrong here.

Weights come as a dict name -> array (already widened to float); `cfg` is the parsed config.json.
"""
from __future__ import annotations

import numpy as np


def linear(w, x, b=None):
    y = x @ w.T
    return y if b is None else y + b


def sigmoid(x):
    return 0.5 * (1.0 + np.tanh(0.5 * x))


def silu(x):
    return x * sigmoid(x)


def relu(x):
    return np.maximum(x, 0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def softplus(x):
    return np.logaddexp(0.0, x)


def rms(x, eps):
    """x over its root mean square, along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rotation(positions, dims, base):
    """cos and sin of p * base^(-2i/dims), [len(positions), dims / 2]."""
    f = float(base) ** (-2.0 * np.arange(dims // 2) / dims)
    a = np.asarray(positions, np.float64)[:, None] * f[None, :]
    return np.cos(a), np.sin(a)


def rotate_half(x, dims, base, first=0):
    """x [T, ..., d]: dimension i turns with dimension i + dims/2 (i < dims/2), the dimensions from `dims` on stay."""
    c, s = rotation(first + np.arange(x.shape[0]), dims, base)
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (dims // 2,)
    c, s = c.reshape(shape), s.reshape(shape)
    y = x.copy()
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    y[..., :dims // 2], y[..., dims // 2:dims] = u * c - v * s, v * c + u * s
    return y


def rotate_pairs(x, dims, base, first=0):
    """The same with dimension 2i turning with dimension 2i + 1."""
    c, s = rotation(first + np.arange(x.shape[0]), dims, base)
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (dims // 2,)
    c, s = c.reshape(shape), s.reshape(shape)
    y = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y[..., 0:dims:2], y[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return y


def retention(q, k, v, decay):
    """One head: q, k [T, dk], v [T, dv] -> o [T, dv], final state [dk, dv]."""
    S = np.zeros((q.shape[1], v.shape[1]))
    o = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay * S + np.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o, S


def retention_mixer(W, p, m, h, eps):
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = rotate_half(linear(W[p + "q"], h).reshape(T, H, dk), m["rot"]["dims"], m["rot"]["base"])
    k = rotate_half(linear(W[p + "k"], h).reshape(T, H, dk), m["rot"]["dims"], m["rot"]["base"]) * dk ** -0.5
    v = linear(W[p + "v"], h).reshape(T, H, dv)
    o = np.stack([retention(q[:, i], k[:, i], v[:, i], m["decay"][i])[0] for i in range(H)], axis=1)
    return linear(W[p + "o"], rms(o, eps).reshape(T, H * dv) * silu(linear(W[p + "g"], h)))


def causal_conv(x, w, b):
    """One filter per channel; the last tap meets the current token, zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return b + sum(pad[j:j + T] * w[:, j] for j in range(taps))


def block_linear(w, b, u):
    """u [T, C] in blocks of w.shape[1] channels, each with a square matrix of its own."""
    T, (n, s, _) = u.shape[0], w.shape
    return (np.einsum("bij,tbj->tbi", w, u.reshape(T, n, s)) + b).reshape(T, n * s)


def rglru(u, r, i, lam):
    """u, r, i [T, C] -> S [T, C]."""
    S, out = np.zeros(u.shape[1]), np.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        S = np.exp(log_a) * S + np.sqrt(-np.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = S
    return out


def rglru_mixer(W, p, m, h):
    y = gelu_tanh(linear(W[p + "y"], h, W[p + "y.b"]))
    u = causal_conv(linear(W[p + "x"], h, W[p + "x.b"]), W[p + "conv"], W[p + "conv.b"])
    r = sigmoid(block_linear(W[p + "ra"], W[p + "ra.b"], u))
    i = sigmoid(block_linear(W[p + "ri"], W[p + "ri.b"], u))
    return linear(W[p + "o"], rglru(u, r, i, W[p + "lam"]) * y)


def window_attention(q, k, v, scale, window):
    """q, k [T, H, d], v [T, H, dv]; position i sees j with 0 <= i - j < window (0: everything up to itself)."""
    T = q.shape[0]
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    mask = (d >= 0) & ((d < window) if window else True)
    out = np.zeros((T, q.shape[1], v.shape[2]))
    for h in range(q.shape[1]):
        s = np.where(mask, (q[:, h] @ k[:, h].T) * scale, -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (e / e.sum(axis=1, keepdims=True)) @ v[:, h]
    return out


def latent_attention_mixer(W, p, m, h, eps):
    T, H, d, r, dv, c = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = linear(W[p + "q"], h).reshape(T, H, d + r)
    lat = linear(W[p + "dkv"], h)
    qr = rotate_pairs(q[..., d:], r, m["rot"]["base"])
    kr = rotate_pairs(lat[:, c:], r, m["rot"]["base"])
    lat = rms(lat[:, :c], eps) * W[p + "dkv.norm"]
    k = linear(W[p + "uk"], lat).reshape(T, H, d)
    v = linear(W[p + "uv"], lat).reshape(T, H, dv)
    k = np.concatenate([k, np.repeat(kr[:, None], H, axis=1)], axis=-1)
    q = np.concatenate([q[..., :d], qr], axis=-1)
    window = (m.get("mask") or {}).get("size", 0)
    o = window_attention(q, k, v, m["scale"], window).reshape(T, H * dv)
    return linear(W[p + "o"], o * sigmoid(linear(W[p + "g"], h)))


def dense_mlp(W, p, h):
    a = relu(linear(W[p + "gate"], h, W[p + "gate.b"])) * linear(W[p + "up"], h, W[p + "up.b"])
    return linear(W[p + "down"], a, W[p + "down.b"])


def route(z, top):
    """Router logits [T, E] -> the chosen experts [T, top] and their scores, which are the weights."""
    s = sigmoid(z)
    chosen = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=1)


def expert(W, p, x):
    return linear(W[p + "down"], silu(linear(W[p + "gate"], x)) * linear(W[p + "up"], x))


def moe_mlp(W, p, m, h):
    chosen, weight = route(linear(W[p + "router"], h), m["router"]["top"])
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t], weight[t]):
            y[t] += expert(W, p + "e%d." % e, w * h[t])
    return y


def forward(cfg, W, tokens, dtype=np.float64):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    W = {n: np.asarray(a, dtype=dtype) for n, a in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    stream = []
    for i, L in enumerate(cfg["layers"]):
        own = i
        while "weights_of" in cfg["layers"][own]:
            own = cfg["layers"][own]["weights_of"]
        p = "l%d." % own
        h = rms(x, eps) * W[p + "norm1"]
        if L["type"] == "retention":
            x = x + retention_mixer(W, p + "mix.", L["mixer"], h, eps)
        elif L["type"] == "rglru":
            x = x + rglru_mixer(W, p + "mix.", L["mixer"], h)
        else:
            x = x + latent_attention_mixer(W, p + "mix.", L["mixer"], h, eps)
        if L.get("mlp"):
            h = rms(x, eps) * W[p + "norm2"]
            x = x + (dense_mlp(W, p + "mlp.", h) if L["mlp"]["kind"] == "dense" else moe_mlp(W, p + "mlp.", L["mlp"], h))
        stream.append(x)
    return linear(W["head"], rms(x, eps) * W["final.norm"]), np.stack(stream)


def greedy(cfg, W, prompt, n_new):
    """n_new greedy tokens after the prompt, and the top-2 margin each was chosen with."""
    toks, out, margins = list(prompt), [], []
    for _ in range(n_new):
        lg = forward(cfg, W, toks)[0][-1]
        s = np.sort(lg)
        margins.append(float(s[-1] - s[-2]))
        out.append(int(np.argmax(lg)))
        toks.append(out[-1])
    return out, margins
