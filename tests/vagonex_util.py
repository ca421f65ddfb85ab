"""Small random Vagonex models for the tests: configurations, weights (exactly representable in bf16), models."""
import numpy as np

from jasmine_b200.decoder import vagonex_model
from zugolorn_util import bf16_bits, error, oracle_weights, run_portions, save_folder, tokens, widen  # noqa: F401


def _layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def attention(heads=4, kv_heads=2, dim=24, vdim=20, rot_dims=12, base=10000.0, scaling=None, size=40, scale=None, kv_from=None, ff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
         "rot": {"base": base, "dims": rot_dims, "scaling": scaling}, "mask": {"size": size} if size else None}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return _layer("attention", m, ff)


def lightning(heads=3, dim=20, vdim=28, decay=None, ff=None):
    decay = decay or [0.5, 0.99, 0.9995, 0.8, 1.0, 0.0, 0.95][:heads]
    return _layer("lightning", {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, ff)


def delta(heads=4, kv_heads=2, dim=24, vdim=20, conv=3, ff=None):
    return _layer("delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, ff)


YARN = {"factor": 4.0, "fast": 16.0, "slow": 2.0, "original": 512}


def config(layers, width=48, vocab=72, alpha=1.5, scale=3.0, eps=1e-5):
    return {"architecture": "Vagonex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "postln_alpha": alpha,
            "embedding": {"scale": scale}, "layers": layers}


def random_weights(cfg, seed, q_gain=1.5):
    """name -> bf16 bits.  q_gain sharpens the attention, so that a single key matters."""
    rng = np.random.default_rng(seed)
    w = {}

    def put(name, shape, std, mean=0.0):
        w[name] = bf16_bits(mean + std * rng.standard_normal(shape))

    d = cfg["width"]
    put("embed", (cfg["vocab"], d), 1.0 / cfg["embedding"]["scale"])
    put("final.norm", (d,), 0.2, 1.0)
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        x, H, n, v = p + "mix.", m["heads"], m["dim"], m["vdim"]
        put(p + "norm1", (d,), 0.2, 1.0)
        if e["type"] == "attention":
            G = m["kv_heads"]
            put(x + "q", (H * n, d), d ** -0.5)
            put(x + "q.b", (H * n,), 0.5)
            put(x + "q.norm", (n,), 0.3, q_gain)
            if m.get("kv_from") is None:
                put(x + "k", (G * n, d), d ** -0.5)
                put(x + "k.b", (G * n,), 0.5)
                put(x + "k.norm", (n,), 0.3, 1.0)
                put(x + "v", (G * v, d), d ** -0.5)
                put(x + "v.b", (G * v,), 0.5)
            put(x + "sink", (H,), 1.0, 1.0)
            put(x + "g", (H, d), 1.5 * d ** -0.5)
        elif e["type"] == "lightning":
            for s, rows in (("q", H * n), ("k", H * n), ("v", H * v), ("g", H * v)):
                put(x + s, (rows, d), 1.5 * d ** -0.5)
            put(x + "norm", (H * v,), 0.3, 1.0)
        else:
            G = m["kv_heads"]
            for s, rows in (("q", G * n), ("k", G * n), ("v", H * v)):
                put(x + s, (rows, d), 1.5 * d ** -0.5)
                put(x + s + ".conv", (rows, m["conv"]), m["conv"] ** -0.5)
            put(x + "b", (H, d), 1.5 * d ** -0.5)
            put(x + "a", (H, d), d ** -0.5)
            put(x + "A_log", (H,), 1.0, -1.5)
            put(x + "dt_bias", (H,), 1.0, -2.0)
            put(x + "g", (H * v, d), 1.5 * d ** -0.5)
            put(x + "norm", (v,), 0.3, 1.0)
        put(x + "o", (d, H * v), (H * v) ** -0.5)
        if e["mlp"] is not None:
            f = e["mlp"]["ff"]
            put(p + "norm2", (d,), 0.2, 1.0)
            put(p + "mlp.gate", (f, d), 1.5 * d ** -0.5)
            put(p + "mlp.up", (f, d), d ** -0.5)
            put(p + "mlp.down", (d, f), f ** -0.5)
    return w


def build(cfg, w, dtype="float32", **serving):
    serving = {"max_batch": 4, "max_context": 1024, "max_step_tokens": 1024, **serving}
    m = vagonex_model(cfg, dtype=dtype, **serving)
    for k, v in w.items():
        m.set_weight(k, v)
    return m.finalize()
