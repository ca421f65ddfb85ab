"""Plain implementation of the Vagonex decoder in numpy float64: one function per mechanism, whole sequences only (no cache, no
state carried between calls).  It shares no code with the library; the GPU tests compare against it.

A model is (config, weights): config has the keys of a config.json, weights maps tensor names to float64 arrays."""
import math

import numpy as np


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(x):
    return 0.5 * (1.0 + np.tanh(0.5 * x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


# ---- rotation ---------------------------------------------------------------------------------------------------------
def yarn(dims, base, scaling):
    """(angle per position of every pair, factor on cos and sin)."""
    freq = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return freq, 1.0
    turns_at = lambda t: dims * math.log(scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(turns_at(scaling["fast"])), 0)
    hi = min(math.ceil(turns_at(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return freq / scaling["factor"] * ramp + freq * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_interleaved(x, positions, freq, magnitude):
    """Pairs (0, 1), (2, 3), ... of the first 2 len(freq) components of the last axis.  x: [T, heads, n]."""
    out = x.copy()
    for i, f in enumerate(freq):
        a = np.asarray(positions, np.float64)[:, None] * f
        c, s = magnitude * np.cos(a), magnitude * np.sin(a)
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ---- attention --------------------------------------------------------------------------------------------------------
def chunked_sink_attention(q, k, v, scale, size, sink):
    """q: [T, H, n], k: [T, G, n], v: [T, G, m]; a query sees the keys before it that lie in its own chunk of `size`
    positions (None: all); exp(sink) of the head joins the denominator."""
    T, H, _ = q.shape
    out = np.empty((T, H, v.shape[2]))
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    seen = j <= i
    if size:
        seen &= i // size == j // size
    for h in range(H):
        g = h // (H // k.shape[1])
        s = np.where(seen, q[:, h] @ k[:, g].T * scale, -np.inf)
        top = np.maximum(s.max(axis=1), sink[h])[:, None]
        e = np.exp(s - top)
        out[:, h] = (e @ v[:, g]) / (e.sum(axis=1, keepdims=True) + np.exp(sink[h] - top))
    return out


def keys_values(x, w, mix, eps):
    T, G, n = x.shape[0], mix["kv_heads"], mix["dim"]
    freq, mag = yarn(mix["rot"]["dims"], mix["rot"]["base"], mix["rot"].get("scaling"))
    k = rms_norm((x @ w["k"].T + w["k.b"]).reshape(T, G, n), w["k.norm"], eps)
    return rotate_interleaved(k, np.arange(T), freq, mag), (x @ w["v"].T + w["v.b"]).reshape(T, G, mix["vdim"])


def attention(x, w, mix, eps, kv=None):
    """w: dict of q, q.b, q.norm, k, k.b, k.norm, v, v.b, sink, g, o; kv: keys and values of another layer.  Returns (out, kv)."""
    T, H, n = x.shape[0], mix["heads"], mix["dim"]
    kv = keys_values(x, w, mix, eps) if kv is None else kv
    freq, mag = yarn(mix["rot"]["dims"], mix["rot"]["base"], mix["rot"].get("scaling"))
    q = rms_norm((x @ w["q"].T + w["q.b"]).reshape(T, H, n), w["q.norm"], eps)
    q = rotate_interleaved(q, np.arange(T), freq, mag)
    o = chunked_sink_attention(q, *kv, mix["scale"], (mix.get("mask") or {}).get("size"), w["sink"])
    o = o * sigmoid(x @ w["g"].T)[:, :, None]
    return o.reshape(T, H * mix["vdim"]) @ w["o"].T, kv


# ---- recurrences ------------------------------------------------------------------------------------------------------
def decayed_sum(q, k, v, decay, state=None):
    """q, k: [T, H, n], v: [T, H, m], decay: [H]; S <- decay S + k v^T, o = S^T q."""
    T, H, n = q.shape
    S = np.zeros((H, n, v.shape[2])) if state is None else state.copy()
    o = np.empty_like(v)
    for t in range(T):
        S = np.asarray(decay)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hnm,hn->hm", S, q[t])
    return o, S


def lightning(x, w, mix, eps):
    """w: dict of q, k, v, g, o, norm."""
    T, H, n, m = x.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    q, k = (silu(x @ w[s].T).reshape(T, H, n) for s in ("q", "k"))
    o, _ = decayed_sum(q, k, silu(x @ w["v"].T).reshape(T, H, m), mix["decay"])
    return (rms_norm(o.reshape(T, H * m), w["norm"], eps) * sigmoid(x @ w["g"].T)) @ w["o"].T


def causal_conv(x, w):
    """Per channel: out[t] = sum_k w[k] x[t - taps + 1 + k].  x: [T, C], w: [C, taps]."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return sum(padded[k:k + x.shape[0]] * w[:, k] for k in range(taps))


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_rule(q, k, v, g, beta, state=None):
    """q, k: [T, H, n], v: [T, H, m], g, beta: [T, H]; S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    T, H, n = q.shape
    S = np.zeros((H, n, v.shape[2])) if state is None else state.copy()
    o = np.empty_like(v)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hnm,hn->hm", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hnm,hn->hm", S, q[t])
    return o, S


def gated_delta(x, w, mix, eps):
    """w: dict of q, k, v (each with .conv), b, a, A_log, dt_bias, norm, g, o."""
    T, H, G, n, m = x.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q, k, v = (silu(causal_conv(x @ w[s].T, w[s + ".conv"])) for s in ("q", "k", "v"))
    q = np.repeat(unit(q.reshape(T, G, n)) * n ** -0.5, H // G, axis=1)
    k = np.repeat(unit(k.reshape(T, G, n)), H // G, axis=1)
    beta = sigmoid(x @ w["b"].T)
    g = np.exp(-np.exp(w["A_log"]) * softplus(x @ w["a"].T + w["dt_bias"]))
    o, _ = delta_rule(q, k, v.reshape(T, H, m), g, beta)
    o = rms_norm(o, w["norm"], eps) * silu(x @ w["g"].T).reshape(T, H, m)
    return o.reshape(T, H * m) @ w["o"].T


# ---- layers -----------------------------------------------------------------------------------------------------------
def gelu_glu(x, w):
    """w: dict of gate, up, down."""
    return (gelu_tanh(x @ w["gate"].T) * (x @ w["up"].T)) @ w["down"].T


def _part(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(config, weights, tokens, residuals=None):
    """Logits of every position, [T, vocab]; appends the residual stream after every layer to `residuals`."""
    eps, alpha = config["norm"]["eps"], config["postln_alpha"]
    x = weights["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    kv = {}
    for i, layer in enumerate(config["layers"]):
        pre, mix = f"l{i}.", layer["mixer"]
        w = _part(weights, pre + "mix.")
        if layer["type"] == "attention":
            y, kv[i] = attention(x, w, mix, eps, None if mix.get("kv_from") is None else kv[mix["kv_from"]])
        elif layer["type"] == "lightning":
            y = lightning(x, w, mix, eps)
        else:
            y = gated_delta(x, w, mix, eps)
        x = rms_norm(alpha * x + y, weights[pre + "norm1"], eps)
        if layer["mlp"] is not None:
            x = rms_norm(alpha * x + gelu_glu(x, _part(weights, pre + "mlp.")), weights[pre + "norm2"], eps)
        if residuals is not None:
            residuals.append(x.copy())
    return rms_norm(x, weights["final.norm"], eps) @ weights["embed"].T
