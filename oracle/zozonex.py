"""Plain restatement of the Zozonex decoder on the host (TEST INFRASTRUCTURE, NOT PRODUCT).

One function per mechanism, written from the equations in float64 numpy with explicit loops over tokens where a
recurrence or a causal mask is involved; it shares no code with the CUDA path.  Sequences are processed whole: there is
no cache, so whatever a cache could get wrong cannot be wrong here.

Weights come as a dict name -> array (already widened to float); `cfg` is the parsed config.json.
"""
from __future__ import annotations

import numpy as np


def linear(w, x):
    return x @ w.T


def silu(x):
    return x / (1.0 + np.exp(-x))


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def softplus(x):
    return np.logaddexp(0.0, x)


def rms(x, eps):
    """x over its root mean square, along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_around_zero(x, w, eps):
    """RMS norm whose stored weight is an offset from one."""
    return rms(x, eps) * (1.0 + w)


def sinusoid(positions, width):
    """Position vectors: sin / cos of p / 10000^(2i/width), interleaved."""
    out = np.zeros((len(positions), width))
    for c in range(width):
        angle = np.asarray(positions, dtype=np.float64) * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = np.sin(angle) if c % 2 == 0 else np.cos(angle)
    return out


def embed(table, tokens, scale):
    x = table[np.asarray(tokens)] * scale
    return x + sinusoid(np.arange(len(tokens)), table.shape[1])


def short_conv(x, w):
    """Causal convolution over time, one filter per channel; the last tap meets the current token."""
    T, C = x.shape
    taps = w.shape[1]
    y = np.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return y


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_decay(a, A_log, dt_bias):
    return np.exp(-np.exp(A_log) * softplus(a + dt_bias))


def delta_rule(q, k, v, g, beta):
    """Gated delta rule of ONE head: q, k [T, dk], v [T, dv], g, beta [T] -> o [T, dv], final state [dk, dv]."""
    T, dk = q.shape
    S = np.zeros((dk, v.shape[1]))
    o = np.zeros_like(v)
    for t in range(T):
        S = g[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        o[t] = S.T @ q[t]
    return o, S


def gated_head_norm(o, gate, w, eps):
    """o [T, heads, dv]: RMS norm per head with one weight vector for all heads, times silu of the gate."""
    return rms(o, eps) * w * silu(gate)


def delta_mixer(W, p, m, h, eps):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(short_conv(linear(W[p + "q"], h), W[p + "q.conv"])).reshape(T, G, dk)
    k = silu(short_conv(linear(W[p + "k"], h), W[p + "k.conv"])).reshape(T, G, dk)
    v = silu(short_conv(linear(W[p + "v"], h), W[p + "v.conv"])).reshape(T, H, dv)
    q = unit(q) * dk ** -0.5
    k = unit(k)
    beta = sigmoid(linear(W[p + "b"], h))
    g = delta_decay(linear(W[p + "a"], h), W[p + "A_log"], W[p + "dt_bias"])
    o = np.zeros((T, H, dv))
    for hd in range(H):
        kv = hd // (H // G)
        o[:, hd], _ = delta_rule(q[:, kv], k[:, kv], v[:, hd], g[:, hd], beta[:, hd])
    gate = linear(W[p + "g"], h).reshape(T, H, dv)
    return linear(W[p + "o"], gated_head_norm(o, gate, W[p + "norm"], eps).reshape(T, H * dv))


def softmax_with_sink(s):
    """exp(s_j) / (1 + sum exp(s_j)) over the last axis; -inf entries have no weight."""
    m = np.maximum(np.max(s, axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (np.exp(-m) + np.sum(e, axis=-1, keepdims=True))


def window_mask(T, size):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (i - j >= 0) & ((i - j < size) if size else True)


def attention(q, k, v, scale, window):
    """q [T, H, dk] against k [T, G, dk], v [T, G, dv] (already normalised)."""
    T, H, _ = q.shape
    G = k.shape[1]
    mask = window_mask(T, window)
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        kv = h // (H // G)
        s = np.where(mask, (q[:, h] @ k[:, kv].T) * scale, -np.inf)
        out[:, h] = softmax_with_sink(s) @ v[:, kv]
    return out


def attention_mixer(W, p, m, h, eps, shared):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(linear(W[p + "q"], h).reshape(T, H, dk), eps)
    if m.get("kv_from") is None:
        k = rms(linear(W[p + "k"], h).reshape(T, G, dk), eps)
        v = linear(W[p + "v"], h).reshape(T, G, dv)
    else:
        k, v = shared[m["kv_from"]]
    window = (m.get("mask") or {}).get("size", 0)
    o = attention(q, k, v, m["scale"], window)
    return linear(W[p + "o"], o.reshape(T, H * dv)), (k, v)


def relu_squared_mlp(W, p, x):
    a = np.maximum(linear(W[p + "up"], x), 0.0)
    return linear(W[p + "down"], a * a)


def forward(cfg, W, tokens, dtype=np.float64):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    W = {n: np.asarray(a, dtype=dtype) for n, a in W.items()}
    eps = cfg["norm"]["eps"]
    x = embed(W["embed"], tokens, cfg["embedding"]["scale"]).astype(dtype)
    shared, stream = {}, []
    for i, L in enumerate(cfg["layers"]):
        p = "l%d." % i
        if L["type"] == "delta":
            y = delta_mixer(W, p + "mix.", L["mixer"], x, eps)
        else:
            y, shared[i] = attention_mixer(W, p + "mix.", L["mixer"], x, eps, shared)
        x = x + norm_around_zero(y, W[p + "norm1"], eps)
        if L.get("mlp"):
            x = x + norm_around_zero(relu_squared_mlp(W, p + "mlp.", x), W[p + "norm2"], eps)
        stream.append(x)
    logits = linear(W["embed"], norm_around_zero(x, W["final.norm"], eps))
    return logits, np.stack(stream)


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
