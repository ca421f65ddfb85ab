"""Plain implementation of the Zugolorn decoder in numpy float64: one function per mechanism, whole sequences only (no
cache, no state carried between calls).  It shares no code with the library; the GPU tests compare against it.

A model is (config, weights): config has the keys of a config.json, weights maps tensor names to float64 arrays."""
import numpy as np


def rms_norm(x, w, eps):
    x = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return x if w is None else x * w


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def rotate_half(x, positions, base):
    """Rotation of the last axis: component i pairs with component i + n/2.  x: [T, ..., n], positions: [T]."""
    n = x.shape[-1]
    freq = float(base) ** (-2.0 * np.arange(n // 2) / n)
    ang = np.asarray(positions, np.float64)[:, None] * freq
    ang = ang.reshape((ang.shape[0],) + (1,) * (x.ndim - 2) + (n // 2,))
    c, s = np.cos(ang), np.sin(ang)
    u, v = x[..., : n // 2], x[..., n // 2:]
    return np.concatenate([u * c - v * s, v * c + u * s], axis=-1)


def window_softmax_attention(q, k, v, scale, window):
    """q, k: [T, H, n], v: [T, H, m]; query i sees the keys i - window + 1 .. i."""
    T = q.shape[0]
    s = np.einsum("ihd,jhd->hij", q, k) * scale
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    seen = (j <= i) & (i - j < window)
    s = np.where(seen[None], s, -np.inf)
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    p = p / p.sum(axis=-1, keepdims=True)
    return np.einsum("hij,jhm->ihm", p, v)


def latent_attention(h, w, mix, eps, positions=None):
    """w: dict of q, dkv, dkv.norm, uk, uv, o."""
    T, H, n, r, m, rank = h.shape[0], mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"], mix["kv_rank"]
    positions = np.arange(T) if positions is None else positions
    base = mix["rot"]["base"]
    q = (h @ w["q"].T).reshape(T, H, n + r)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :rank], w["dkv.norm"], eps)
    kr = rotate_half(down[:, None, rank:], positions, base)
    k = np.concatenate([(c @ w["uk"].T).reshape(T, H, n), np.broadcast_to(kr, (T, H, r))], axis=-1)
    v = (c @ w["uv"].T).reshape(T, H, m)
    q = np.concatenate([q[..., :n], rotate_half(q[..., n:], positions, base)], axis=-1)
    return window_softmax_attention(q, k, v, mix["scale"], mix["mask"]["size"]).reshape(T, H * m) @ w["o"].T


def causal_conv(x, w, b):
    """Per channel: out[t] = b + sum_k w[k] x[t - taps + 1 + k].  x: [T, C], w: [C, taps]."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return sum(padded[k:k + x.shape[0]] * w[:, k] for k in range(taps)) + b


def selective_scan(x, dt, A, B, C, D, state=None):
    """x, dt: [T, inner]; A: [inner, n]; B, C: [T, n].  Returns (y, final state)."""
    S = np.zeros(A.shape) if state is None else state.copy()
    y = np.empty_like(x)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def mamba1(h, w, mix):
    """w: dict of in, conv, conv.b, x, dt, dt.b, A_log, D, o."""
    inner, n, R = mix["inner"], mix["state"], mix["dt_rank"]
    xz = h @ w["in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, w["conv"], w["conv.b"]))
    p = x @ w["x"].T
    dt = softplus(p[:, :R] @ w["dt"].T + w["dt.b"])
    y, _ = selective_scan(x, dt, -np.exp(w["A_log"]), p[:, R:R + n], p[:, R + n:], w["D"])
    return (y * silu(z)) @ w["o"].T


def clamped_glu(h, w, limit):
    """w: dict of gate, up, down."""
    g = np.minimum(h @ w["gate"].T, limit)
    u = np.clip(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w["down"].T


def softcap(x, cap):
    return cap * np.tanh(x / cap)


def _part(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(config, weights, tokens, residuals=None):
    """Logits of every position, [T, vocab]; appends the residual stream after every layer to `residuals`."""
    eps = config["norm"]["eps"]
    x = weights["embed"][np.asarray(tokens)]
    for i, layer in enumerate(config["layers"]):
        pre = f"l{layer.get('weights_of', i)}."
        w = _part(weights, pre + "mix.")
        if layer["type"] == "latent_attention":
            y = latent_attention(x, w, layer["mixer"], eps)
        else:
            y = mamba1(x, w, layer["mixer"])
        x = x + rms_norm(y, weights[pre + "norm1"], eps)
        if layer["mlp"] is not None:
            y = clamped_glu(x, _part(weights, pre + "mlp."), layer["mlp"]["limit"])
            x = x + rms_norm(y, weights[pre + "norm2"], eps)
        if residuals is not None:
            residuals.append(x.copy())
    return softcap(rms_norm(x, weights["final.norm"], eps) @ weights["embed"].T, config["logit_softcap"])
