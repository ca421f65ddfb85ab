"""Small random Zugolorn models for the tests: configurations, weights (exactly representable in bf16), model folders."""
import json

import numpy as np

from jasmine_b200.decoder import zugolorn_model


def bf16_bits(x):
    u = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def widen(bits):
    return (bits.astype(np.uint32) << 16).view(np.float32).astype(np.float64)


def attention(heads=3, dim=16, rot_dim=8, vdim=12, kv_rank=20, window=40, base=10000.0, scale=None, ff=None, limit=1.5):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
                      "rot": {"base": base, "dims": rot_dim}, "scale": scale or (dim + rot_dim) ** -0.5},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def mamba(inner=48, state=5, dt_rank=3, conv=4, ff=None, limit=1.5):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def shared(config_layers, j):
    e = json.loads(json.dumps(config_layers[j]))
    e["weights_of"] = j
    return e


def config(layers, width=40, vocab=72, cap=6.0, eps=1e-5):
    return {"architecture": "Zugolorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}


def random_weights(cfg, seed, q_gain=1.5, norm_gain=0.4):
    """name -> bf16 bits.  q_gain sharpens the attention, so that a single key matters; norm_gain below 1 keeps the residual
    stream from amplifying roundings layer after layer."""
    rng = np.random.default_rng(seed)
    w = {}

    def put(name, shape, std, mean=0.0):
        w[name] = bf16_bits(mean + std * rng.standard_normal(shape))

    d = cfg["width"]
    put("embed", (cfg["vocab"], d), 1.0)
    put("final.norm", (d,), 0.2, 1.0)
    for i, e in enumerate(cfg["layers"]):
        if "weights_of" in e:
            continue
        p, m = f"l{i}.", e["mixer"]
        put(p + "norm1", (d,), 0.2 * norm_gain, norm_gain)
        if e["type"] == "latent_attention":
            H, r = m["heads"], m["kv_rank"]
            put(p + "mix.q", (H * (m["dim"] + m["rot_dim"]), d), q_gain * d ** -0.5)
            put(p + "mix.dkv", (r + m["rot_dim"], d), d ** -0.5)
            put(p + "mix.dkv.norm", (r,), 0.2, 1.0)
            put(p + "mix.uk", (H * m["dim"], r), r ** -0.5)
            put(p + "mix.uv", (H * m["vdim"], r), r ** -0.5)
            put(p + "mix.o", (d, H * m["vdim"]), (H * m["vdim"]) ** -0.5)
        else:
            c, n, R = m["inner"], m["state"], m["dt_rank"]
            put(p + "mix.in", (2 * c, d), d ** -0.5)
            put(p + "mix.conv", (c, m["conv"]), m["conv"] ** -0.5)
            put(p + "mix.conv.b", (c,), 0.3)
            put(p + "mix.x", (R + 2 * n, c), 1.5 * c ** -0.5)
            put(p + "mix.dt", (c, R), R ** -0.5)
            put(p + "mix.dt.b", (c,), 0.7, -2.0)
            put(p + "mix.A_log", (c, n), 0.7)
            put(p + "mix.D", (c,), 0.5, 0.5)
            put(p + "mix.o", (d, c), c ** -0.5)
        if e["mlp"] is not None:
            f = e["mlp"]["ff"]
            put(p + "norm2", (d,), 0.2 * norm_gain, norm_gain)
            put(p + "mlp.gate", (f, d), d ** -0.5)
            put(p + "mlp.up", (f, d), d ** -0.5)
            put(p + "mlp.down", (d, f), f ** -0.5)
    return w


def oracle_weights(w):
    return {k: widen(v) for k, v in w.items()}


def build(cfg, w, dtype="float32", **serving):
    serving = {"max_batch": 4, "max_context": 1024, "max_step_tokens": 1024, **serving}
    m = zugolorn_model(cfg, dtype=dtype, **serving)
    for k, v in w.items():
        m.set_weight(k, v)
    return m.finalize()


def save_folder(folder, cfg, w):
    (folder / "config.json").write_text(json.dumps(cfg))
    header, at = {}, 0
    for k, v in w.items():
        header[k] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [at, at + v.nbytes]}
        at += v.nbytes
    head = json.dumps(header).encode()
    with open(folder / "model.safetensors", "wb") as f:
        f.write(len(head).to_bytes(8, "little") + head)
        for v in w.values():
            f.write(v.tobytes())


def tokens(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def error(got, want):
    """Worst row: rms difference (means taken off) over the rms of the wanted logits."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    w = want - want.mean(axis=-1, keepdims=True)
    return float(np.sqrt((d * d).mean(axis=-1)).max() / np.sqrt((w * w).mean()))


def run_portions(m, toks, sizes, row=None):
    """Logits of every position, the tokens brought in portions of the given sizes (the last size repeats)."""
    own = row is None
    row = m.open() if own else row
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - at)
        _, lg = m.step([(row, toks[at:at + n])], range(n))
        out.append(lg)
        at += n
        k += 1
    if own:
        m.retire(row)
    return np.concatenate(out)
