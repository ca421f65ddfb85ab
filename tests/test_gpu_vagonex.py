"""Vagonex on the GPU against the plain float64 implementation (vagonex_oracle.py): each mechanism alone, prompts, portions,
decoding, batches, reuse of pages and slots, chunk edges, shared keys and values, generation through the scheduler and the
command line.

fp32 models are compared sharply (fp32 rounding only), bf16 models at a bf16 bar; where random weights would hide a fault,
one key, one token or one sink is made to stand out."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import jasmine_b200 as jb
import vagonex_oracle as vo
import vagonex_util as vu
from gpu_util import BF16_RTOL, assert_close
from jasmine_b200 import generate

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
DTYPES = ["float32", "bfloat16"]
TOL = {"float32": 4e-5, "bfloat16": 0.08}


def want_logits(cfg, w, toks):
    return vo.forward(cfg, vu.oracle_weights(w), toks)


# ---- token-level parts ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,N,K", [(1, 64, 64), (5, 200, 40), (24, 328, 64), (40, 64, 520), (64, 1000, 72), (100, 136, 200), (300, 264, 96)])
def test_gelu_gate_up_projection(T, N, K):
    g = torch.Generator(device="cuda").manual_seed(T * 1000 + N)
    x = torch.randn(T, K, device="cuda", generator=g).bfloat16()
    w = (torch.randn(2 * N, K, device="cuda", generator=g) * 2 * K ** -0.5).bfloat16()
    out = torch.empty(T, N, dtype=torch.bfloat16, device="cuda")
    jb.linear_bf16_packed(x, jb.linear_pack(w, N, True), out, epilogue=6)
    y = (x.double() @ w.double().T).cpu().numpy()
    assert_close(out.float().cpu().numpy(), vo.gelu_tanh(y[:, :N]) * y[:, N:], BF16_RTOL / 2)
    jb.check_device_errors()


@pytest.mark.parametrize("T,d,alpha", [(1, 8, 1.0), (3, 40, 2.5), (7, 1000, 0.3), (5, 2048, 3.0), (4, 4096, 1.7), (2, 5000, 4.0)])
def test_norm_of_the_sum(T, d, alpha):
    rng = np.random.default_rng(d)
    y, x, g = (rng.standard_normal(s).astype(np.float32) for s in ((T, d), (T, d), (d,)))
    want = vo.rms_norm(np.float32(alpha) * x.astype(np.float64) + y, g.astype(np.float64), 1e-3)
    xd, xb = torch.from_numpy(x).cuda(), torch.empty(T, d, dtype=torch.bfloat16, device="cuda")
    jb.sum_norm(torch.from_numpy(y).cuda(), xd, torch.from_numpy(g).cuda(), 1e-3, alpha, xb)
    assert_close(xd.cpu().numpy(), want, 1e-6)
    assert torch.equal(xb, xd.bfloat16())


@pytest.mark.parametrize("dims,base,scaling", [(2, 100.0, None), (64, 10000.0, vu.YARN), (24, 500.0, {"factor": 2.0, "fast": 32.0, "slow": 1.0, "original": 4096}),
                                               (6, 10000.0, {"factor": 8.0, "fast": 1.0, "slow": 1.0, "original": 64}), (10, 50.0, {"factor": 1.0, "fast": 4.0, "slow": 3.9, "original": 300})])
def test_scaled_rotation_tables(dims, base, scaling):
    t = torch.empty(700, dims // 2, 2, device="cuda")
    s = scaling or {"factor": 0.0, "original": 0.0, "fast": 0.0, "slow": 0.0}
    jb.check(jb.lib().jsm_rope_scaled_table(t.data_ptr(), dims, base, s["factor"], float(s["original"]), s["fast"], s["slow"], 700))
    freq, mag = vo.yarn(dims, base, scaling)
    ang = np.arange(700)[:, None] * freq
    assert_close(t.cpu().numpy(), mag * np.stack([np.cos(ang), np.sin(ang)], -1), 1e-6)


# ---- mixers alone -----------------------------------------------------------------------------------------------------
def layer_residual(m, toks, sizes):
    """Residual stream after every layer, the tokens brought in portions."""
    row, at, out = m.open(), 0, []
    for n in sizes:
        n = min(n, len(toks) - at)
        if n <= 0:
            break
        buf = torch.zeros(m.n_layers, n, m.d_model, device="cuda")
        m.set_tap(buf)
        m.step([(row, toks[at:at + n])])
        out.append(buf.cpu().numpy())
        at += n
    m.set_tap(None)
    m.retire(row)
    return np.concatenate(out, axis=1)


def mixer_alone(layer, dtype, n=170, seed=3, portions=None, tol=BF16_RTOL, **kw):
    cfg = vu.config([layer], alpha=0.6, **kw)  # (a small alpha: the mixer's share of the sum shows)
    w = vu.random_weights(cfg, seed)
    toks = vu.tokens(n, cfg["vocab"], seed + 1)
    want = []
    vo.forward(cfg, vu.oracle_weights(w), toks, want)
    m = vu.build(cfg, w, dtype)
    for sizes in portions or ([n], [70, 2, 50, n], [1] * 20 + [97] + [1] * n, [129, 3, 1, n], [2, 3, 31, 1, 1, 64, n]):
        got = layer_residual(m, toks, sizes)[0]
        if dtype == "float32":
            assert_close(got, want[0], 1.5e-5, str(sizes[:5]))
        else:  # (a token whose mixer output is tiny before its norm, or whose key is nearly zero, amplifies roundings)
            assert np.sqrt(np.mean((got - want[0]) ** 2) / np.mean(want[0] ** 2)) < 0.8 * tol and vu.error(got, want[0]) < 6 * tol, sizes[:5]
    m.close()


ATTENTION = [dict(), dict(heads=1, kv_heads=1, dim=2, vdim=3, rot_dims=2, size=1), dict(heads=5, kv_heads=5, dim=9, vdim=13, rot_dims=6, size=7),
             dict(heads=6, kv_heads=3, dim=40, vdim=64, rot_dims=40, size=64, scaling=vu.YARN), dict(heads=7, kv_heads=1, dim=64, vdim=24, rot_dims=0, size=65),
             dict(heads=8, kv_heads=2, dim=80, vdim=130, rot_dims=20, size=None), dict(heads=24, kv_heads=2, dim=16, vdim=16, rot_dims=16, size=100, base=300.0),
             dict(heads=9, kv_heads=1, dim=130, vdim=70, rot_dims=64, size=33), dict(heads=2, kv_heads=2, dim=200, vdim=200, rot_dims=100, size=128, scaling=vu.YARN),
             dict(heads=4, kv_heads=1, dim=300, vdim=280, rot_dims=64, size=50), dict(heads=16, kv_heads=1, dim=128, vdim=128, rot_dims=128, size=96, scale=0.2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", ATTENTION, ids=lambda k: "-".join(str(v) for v in k.values() if not isinstance(v, dict)) or "default")
def test_attention_alone(kw, dtype):
    mixer_alone(vu.attention(**kw), dtype)


LIGHTNING = [dict(), dict(heads=1, dim=1, vdim=3, decay=[0.9]), dict(heads=7, dim=9, vdim=17), dict(heads=2, dim=64, vdim=64), dict(heads=2, dim=128, vdim=64, decay=[0.999, 0.3]),
             dict(heads=2, dim=64, vdim=128, decay=[0.97, 1.0]), dict(heads=2, dim=100, vdim=120), dict(heads=1, dim=200, vdim=200, decay=[0.98]),
             dict(heads=2, dim=32, vdim=260), dict(heads=2, dim=16, vdim=16, decay=[0.0, 0.9])]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", LIGHTNING, ids=lambda k: "-".join(map(str, k.values())) or "default")
def test_decayed_sum_alone(kw, dtype):
    mixer_alone(vu.lightning(**kw), dtype, seed=13)


DELTA = [dict(), dict(heads=1, kv_heads=1, dim=12, vdim=3, conv=1), dict(heads=6, kv_heads=3, dim=9, vdim=17, conv=2), dict(heads=4, kv_heads=1, dim=64, vdim=64, conv=5),
         dict(heads=2, kv_heads=2, dim=128, vdim=128, conv=4), dict(heads=2, kv_heads=1, dim=100, vdim=72, conv=4), dict(heads=3, kv_heads=1, dim=32, vdim=96, conv=3),
         dict(heads=1, kv_heads=1, dim=200, vdim=200, conv=4), dict(heads=2, kv_heads=1, dim=16, vdim=260, conv=7), dict(heads=2, kv_heads=2, dim=128, vdim=64, conv=2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", DELTA, ids=lambda k: "-".join(map(str, k.values())) or "default")
def test_delta_rule_alone(kw, dtype):
    mixer_alone(vu.delta(**kw), dtype, seed=23)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [vu.lightning(heads=2, dim=64, vdim=48), vu.delta(heads=2, kv_heads=1, dim=64, vdim=48), vu.delta(heads=2, kv_heads=1, dim=128, vdim=128)],
                         ids=["decayed", "delta", "delta128"])
def test_recurrences_over_long_prompts(layer, dtype):
    """Many chunks in a row, portions that end on, just before and just behind a chunk's edge."""
    mixer_alone(layer, dtype, n=900, seed=33, width=64, portions=([900], [64, 128, 63, 65, 1, 2, 200, 900], [333, 1, 1, 566], [880] + [1] * 20))


FLASH = [dict(heads=2, kv_heads=1, dim=40, vdim=64), dict(heads=3, kv_heads=3, dim=64, vdim=100), dict(heads=4, kv_heads=2, dim=100, vdim=30),
         dict(heads=2, kv_heads=2, dim=128, vdim=128), dict(heads=3, kv_heads=1, dim=160, vdim=60), dict(heads=2, kv_heads=1, dim=192, vdim=128)]


@pytest.mark.parametrize("size", [20, 128, 200, 257, 2000, None])
@pytest.mark.parametrize("kw", FLASH, ids=lambda k: "-".join(map(str, k.values())))
def test_long_prompts_take_the_flash_kernel(kw, size):
    """Segments of at least 128 tokens; every tile shape, chunks shorter and longer than a tile, portions that start inside a
    page, a tile and a chunk."""
    mixer_alone(vu.attention(rot_dims=16, size=size, **kw), "bfloat16", n=700, seed=31, width=64, tol=1.5 * BF16_RTOL,
                portions=([700], [129, 300, 700], [37, 400, 3, 700], [690] + [1] * 10))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_contexts_are_split_over_the_pages(dtype):
    """One sequence, full mask: few rows and many pages, so that several CTAs share them; a batch of two has fewer splits."""
    cfg = vu.config([vu.attention(heads=4, kv_heads=2, dim=64, vdim=40, rot_dims=32, size=None)], width=64, alpha=0.6)
    w = vu.random_weights(cfg, 41, q_gain=3.0)
    seqs = [vu.tokens(1500, cfg["vocab"], 42), vu.tokens(130, cfg["vocab"], 43)]
    want = [want_logits(cfg, w, s) for s in seqs]
    m = vu.build(cfg, w, dtype, max_context=1536, max_step_tokens=1536)
    got = vu.run_portions(m, seqs[0], [1470, 1, 1, 1, 2, 3, 1])
    assert vu.error(got, want[0]) < TOL[dtype]
    rows = [m.open(), m.open()]
    m.step([(r, s[:-5]) for r, s in zip(rows, seqs)])
    for k in range(5, 0, -1):
        _, lg = m.step([(r, [s[-k]]) for r, s in zip(rows, seqs)], [0, 1])
        for i in range(2):
            assert vu.error(lg[i:i + 1], want[i][len(seqs[i]) - k][None]) < TOL[dtype]
    m.close()


# ---- mechanisms made to stand out -------------------------------------------------------------------------------------
def standing_key_model(size, dtype, layers=1):
    """Every query asks for the key token (token 0 of the vocabulary), whose score exceeds all others by 8."""
    ls = [vu.attention(heads=2, kv_heads=1, dim=16, vdim=16, rot_dims=2, size=size, scale=0.5)]
    ls += [vu.attention(heads=2, kv_heads=1, dim=16, vdim=16, rot_dims=2, size=s, scale=0.5, kv_from=0) for s in ([size * 2] if layers > 1 else [])]
    cfg = vu.config(ls, width=48, alpha=0.5)
    w = vu.random_weights(cfg, 21)
    rng = np.random.default_rng(5)
    emb = vu.widen(w["embed"]).reshape(-1, 48) * 0.3
    emb[:, 0], emb[:, 1] = 1.0, 0.0
    emb[0, 0], emb[0, 1] = 0.0, 1.0
    w["embed"] = vu.bf16_bits(emb)
    k = np.zeros((16, 48))
    k[4, 1], k[5, 0] = 4.0, 4.0
    w["l0.mix.k"], w["l0.mix.k.b"] = vu.bf16_bits(k), vu.bf16_bits(0.01 * rng.standard_normal(16))
    for i in range(len(ls)):
        q = np.zeros((32, 48))
        b = 0.01 * rng.standard_normal(32)
        b[[4, 20]] = 4.0
        w.update({f"l{i}.mix.q": vu.bf16_bits(q), f"l{i}.mix.q.b": vu.bf16_bits(b), f"l{i}.mix.q.norm": vu.bf16_bits(np.ones(16)),
                  f"l{i}.mix.sink": vu.bf16_bits(np.array([0.0, 4.0]))})
    w["l0.mix.k.norm"] = vu.bf16_bits(np.ones(16))
    return cfg, w, vu.build(cfg, w, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [1, 2, 63, 64, 65, 100, 128, 129, 200])
def test_edges_of_a_chunk(size, dtype):
    """The key token is the last one of a chunk, the first of one, or in the middle: it shows to the end of its chunk and not
    one token further, wherever the prompt is cut."""
    cfg, w, m = standing_key_model(size, dtype)
    tol = TOL[dtype]
    for place in (0, size - 1, size, 2 * size + size // 2):
        edge = (place // size + 1) * size  # first position that does not see it
        toks = [1 + t % 71 for t in vu.tokens(max(edge, place) + 150, 71, 30 + place)]
        toks[place] = 0
        want = want_logits(cfg, w, toks)
        other = json.loads(json.dumps(cfg))
        other["layers"][0]["mixer"]["mask"]["size"] = edge + 1  # one position more sees it
        assert vu.error(want_logits(other, w, toks)[edge:edge + 1], want[edge:edge + 1]) > 2 * TOL["bfloat16"]  # the edge shows
        for sizes in ([len(toks)], [max(1, edge - 1), 1, 1, 2], [edge, 130], [max(1, edge - 2), 2, 2], [1] * 3 + [max(1, edge)] + [1], [130, 1]):
            got = vu.run_portions(m, toks, sizes)
            assert vu.error(got[edge - 1:edge + 2], want[edge - 1:edge + 2]) < tol, (place, sizes[:3])
            assert vu.error(got, want) < tol
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_keys_and_values_of_another_layer(dtype):
    """A layer with the keys of an earlier one, but a wider mask of its own: pages stay until the widest mask has left them."""
    cfg, w, m = standing_key_model(50, dtype, layers=2)
    toks = [1 + t % 71 for t in vu.tokens(330, 71, 9)]
    toks[10] = toks[130] = toks[260] = 0
    want = want_logits(cfg, w, toks)
    narrow = json.loads(json.dumps(cfg))
    narrow["layers"][1]["mixer"]["mask"]["size"] = 50
    assert vu.error(want_logits(narrow, w, toks)[60:61], want[60:61]) > 2 * TOL["bfloat16"]
    for sizes in ([330], [99, 1, 1, 99, 130], [1], [2, 40], [200, 2]):
        assert vu.error(vu.run_portions(m, toks, sizes), want) < TOL[dtype], sizes
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink", [-30.0, 0.0, 6.0, 60.0])
def test_sinks_of_every_strength(sink, dtype):
    cfg = vu.config([vu.attention(heads=4, kv_heads=2, dim=32, vdim=32, rot_dims=8, size=90)], alpha=0.5)
    w = vu.random_weights(cfg, 71)
    without = want_logits(cfg, {**w, "l0.mix.sink": vu.bf16_bits(np.full(4, -1000.0))}, vu.tokens(300, 72, 72))
    w["l0.mix.sink"] = vu.bf16_bits(np.array([sink, sink, 0.0, sink]))
    toks = vu.tokens(300, 72, 72)
    want = want_logits(cfg, w, toks)
    assert vu.error(without, want) > 2 * TOL["bfloat16"]
    m = vu.build(cfg, w, dtype)
    for sizes in ([300], [20, 1], [50, 100, 3]):
        assert vu.error(vu.run_portions(m, toks, sizes), want) < TOL[dtype]
    m.close()


def far_token(cfg, w, dtype, n=500):
    """The first token differs from all others; its trace in the state must survive to the end."""
    toks = [2 + t % 70 for t in vu.tokens(n, 70, 8)]
    toks[0] = 0
    want = want_logits(cfg, w, toks)
    assert vu.error(want_logits(cfg, w, [1] + toks[1:])[-1:], want[-1:]) > 2 * TOL["bfloat16"]
    m = vu.build(cfg, w, dtype)
    for sizes in ([n], [150, 2, 1, 200, n], [n - 30] + [1] * 30, [3]):
        assert vu.error(vu.run_portions(m, toks, sizes)[-1:], want[-1:]) < TOL[dtype], sizes[:3]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_decayed_sum_remembers_the_first_token(dtype):
    cfg = vu.config([vu.lightning(heads=2, dim=32, vdim=32, decay=[0.9999, 0.998])], alpha=0.2)
    w = vu.random_weights(cfg, 51)
    emb = vu.widen(w["embed"]).reshape(72, 48)
    emb[:2] *= 8.0  # tokens 0 and 1 write strongly
    w["embed"] = vu.bf16_bits(emb)
    far_token(cfg, w, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_remembers_the_first_token(dtype):
    cfg = vu.config([vu.delta(heads=2, kv_heads=1, dim=64, vdim=32, conv=4)], alpha=0.2)
    w = vu.random_weights(cfg, 61)
    emb = vu.widen(w["embed"]).reshape(72, 48)
    emb[:, 0] = 1.0
    emb[:2, 0] = -1.0
    b = np.zeros((2, 48))
    b[:, 0] = -3.0  # beta: nearly 1 for tokens 0 and 1, nearly 0 for all others
    w.update({"embed": vu.bf16_bits(emb), "l0.mix.b": vu.bf16_bits(b), "l0.mix.A_log": vu.bf16_bits(np.full(2, -9.0))})
    far_token(cfg, w, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_with_keys_that_repeat(dtype):
    """The same token over and over, beta near 1: every write takes back the one before it, the chunk's triangular system is as
    full as it gets; then two tokens in turn, and others."""
    cfg = vu.config([vu.delta(heads=2, kv_heads=1, dim=32, vdim=32, conv=1)], alpha=0.4)
    w = vu.random_weights(cfg, 65)
    emb = vu.widen(w["embed"]).reshape(72, 48)
    emb[:, 0] = 1.0
    b = np.zeros((2, 48))
    b[0, 0], b[1, 0] = 3.0, 1.0  # (x is three times the table)
    w.update({"embed": vu.bf16_bits(emb), "l0.mix.b": vu.bf16_bits(b), "l0.mix.A_log": vu.bf16_bits(np.array([-9.0, -3.0]))})
    toks = [5] * 150 + [6, 7] * 60 + vu.tokens(90, 72, 66)
    want = want_logits(cfg, w, toks)
    m = vu.build(cfg, w, dtype)
    for sizes in ([360], [100, 1, 2, 257], [3]):
        assert vu.error(vu.run_portions(m, toks, sizes), want) < TOL[dtype], sizes
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_decays_from_nothing_to_everything(dtype):
    """Steps that forget the whole state beside steps that keep it: running sums of their logarithms must not drown the rest."""
    cfg = vu.config([vu.delta(heads=2, kv_heads=1, dim=32, vdim=32, conv=2)], alpha=0.4)
    w = vu.random_weights(cfg, 67)
    emb = vu.widen(w["embed"]).reshape(72, 48)
    emb[:, 0] = 0.0
    emb[:4, 0] = 10.0  # tokens 0 .. 3 forget
    a = np.zeros((2, 48))
    a[:, 0] = 3.0
    w.update({"embed": vu.bf16_bits(emb), "l0.mix.a": vu.bf16_bits(a), "l0.mix.A_log": vu.bf16_bits(np.array([2.0, 1.0])),
              "l0.mix.dt_bias": vu.bf16_bits(np.array([-7.0, -8.0]))})
    toks = vu.tokens(300, 72, 68)
    want = want_logits(cfg, w, toks)
    m = vu.build(cfg, w, dtype)
    for sizes in ([300], [64, 7, 1], [1]):
        assert vu.error(vu.run_portions(m, toks, sizes), want) < TOL[dtype], sizes
    m.close()


# ---- whole models -----------------------------------------------------------------------------------------------------
def mixed_config():
    layers = [vu.delta(ff=88), vu.lightning(heads=2, dim=24, vdim=16, ff=40), vu.attention(heads=6, kv_heads=3, size=50, scaling=vu.YARN, ff=56),
              vu.delta(heads=3, kv_heads=1, dim=32, vdim=24, conv=4), vu.attention(heads=6, kv_heads=3, size=90, scaling=vu.YARN, kv_from=2, ff=24),
              vu.attention(heads=5, kv_heads=1, dim=40, vdim=64, rot_dims=40, base=500.0, size=33)]
    return vu.config(layers, width=52, vocab=101, alpha=2.2, scale=5.0)


CFG = mixed_config()
W = vu.random_weights(CFG, 11)


@pytest.fixture(scope="module", params=DTYPES)
def model(request):
    m = vu.build(CFG, W, request.param, max_batch=6)
    m.dtype_name = request.param
    yield m
    m.close()


@pytest.fixture(scope="module")
def long_case():
    toks = vu.tokens(330, CFG["vocab"], 12)
    return toks, want_logits(CFG, W, toks)


def test_residual_stream_after_every_layer(model, long_case):
    want = []
    vo.forward(CFG, vu.oracle_weights(W), long_case[0], want)
    for sizes in ([330], [100, 1, 229]):
        got = layer_residual(model, long_case[0], sizes)
        for a, b in zip(got, want):
            assert_close(a, b, 3e-5 if model.dtype_name == "float32" else 3 * BF16_RTOL)


@pytest.mark.parametrize("sizes", [[330], [1], [2], [3, 5, 7], [64], [63, 65], [130, 1, 1, 140], [200, 2], [33, 50, 90]], ids=str)
def test_portions_of_a_prompt(model, long_case, sizes):
    toks, want = long_case
    assert vu.error(vu.run_portions(model, toks, sizes), want) < TOL[model.dtype_name]


def test_first_tokens(model):
    for n in (1, 2, 3, 4, 5):
        toks = vu.tokens(n, CFG["vocab"], 40 + n)
        want = want_logits(CFG, W, toks)
        for sizes in ([n], [1]):
            assert vu.error(vu.run_portions(model, toks, sizes), want) < TOL[model.dtype_name]


def test_batches_of_unequal_requests(model):
    """Prompts, portions and single tokens of several sequences in one step: each as if it were alone."""
    tol = TOL[model.dtype_name]
    seqs = [vu.tokens(n, CFG["vocab"], 60 + n) for n in (260, 17, 140, 1, 75)]
    want = [want_logits(CFG, W, s) for s in seqs]
    plan = [[250, 9, 2, 1, 40], [1, 1, 130, 0, 1], [1, 1, 1, 0, 30], [2, 1, 1, 0, 1], [1, 1, 1, 0, 1], [1, 4, 5, 0, 2]]
    rows, at = [model.open() for _ in seqs], [0] * 5
    for counts in plan:
        entries, where = [], []
        for i, n in enumerate(counts):
            n = min(n, len(seqs[i]) - at[i])
            if n > 0:
                entries.append((rows[i], seqs[i][at[i]:at[i] + n]))
                where += [(i, at[i] + k) for k in range(n)]
                at[i] += n
        order = np.random.default_rng(len(where)).permutation(len(where))  # the wanted places in any order
        nxt, lg = model.step(entries, order)
        for k, o in enumerate(order):
            i, p = where[o]
            assert vu.error(lg[k:k + 1], want[i][p:p + 1]) < tol, (i, p)
            assert nxt[k] == int(np.argmax(lg[k]))
    for _ in rows:
        model.retire(0)
    assert model.pool_state()[0] == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_slots_are_used_again(dtype):
    """A pool too small for all sequences at once, rows that move, masks that give pages back while a sequence runs."""
    m = vu.build(CFG, W, dtype, max_batch=3, max_context=512, max_step_tokens=96, pool_pages=11)
    seqs = {k: vu.tokens(n, CFG["vocab"], 80 + k) for k, n in enumerate((400, 90, 200, 30, 150))}
    want = {k: want_logits(CFG, W, s) for k, s in seqs.items()}
    rows, at, todo = [], {}, [0, 1, 2, 3, 4]

    def advance(k, n):
        n = min(n, len(seqs[k]) - at[k])
        _, lg = m.step([(rows.index(k), seqs[k][at[k]:at[k] + n])], range(n))
        assert vu.error(lg, want[k][at[k]:at[k] + n]) < TOL[dtype], (k, at[k])
        at[k] += n

    turn = 0
    while todo or rows:
        while todo and len(rows) < 2 + turn % 2:
            k = todo.pop(0)
            assert m.open() == len(rows)
            rows.append(k)
            at[k] = 0
        for k in list(rows):
            advance(k, (70, 1, 33, 2)[turn % 4])
            turn += 1
        for k in list(rows):
            if at[k] == len(seqs[k]):
                i = rows.index(k)
                moved = m.retire(i)
                last = rows.pop()
                if moved >= 0:
                    rows[i] = last
    assert m.pool_state() == (0, 11, 11)  # every page is back
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_kind_of_mixer_only(dtype):
    for layers in ([vu.delta(ff=24), vu.lightning()], [vu.attention(ff=24), vu.attention(size=9)], [vu.attention(size=None)]):
        cfg = vu.config(layers)
        w = vu.random_weights(cfg, 51)
        m = vu.build(cfg, w, dtype, max_batch=2, max_context=100)
        for seed in (52, 53):
            toks = vu.tokens(90, cfg["vocab"], seed)
            assert vu.error(vu.run_portions(m, toks, [60, 2, 1]), want_logits(cfg, w, toks)) < TOL[dtype]
        assert generate.generate(m, [toks[:5], toks[:30]], 4)[0]
        m.close()


def test_steps_longer_than_a_pass_are_cut():
    m = vu.build(CFG, W, "float32", max_step_tokens=50)
    toks = vu.tokens(233, CFG["vocab"], 90)
    assert vu.error(vu.run_portions(m, toks, [233]), want_logits(CFG, W, toks)) < TOL["float32"]
    m.close()


def test_long_decoding(model):
    toks = vu.tokens(420, CFG["vocab"], 91)
    assert vu.error(vu.run_portions(model, toks, [20, 1]), want_logits(CFG, W, toks)) < TOL[model.dtype_name]


# ---- generation -------------------------------------------------------------------------------------------------------
def greedy(cfg, w, prompt, n):
    seq = list(prompt)
    ow = vu.oracle_weights(w)
    for _ in range(n):
        seq.append(int(np.argmax(vo.forward(cfg, ow, seq)[-1])))
    return seq[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    prompts = [vu.tokens(n, CFG["vocab"], 100 + n) for n in (5, 70, 1, 33, 18)]
    lens = [12, 6, 15, 3, 9]
    want = [greedy(CFG, W, p, n) for p, n in zip(prompts, lens)]
    m = vu.build(CFG, W, "float32", max_batch=3, max_context=128, pool_pages=8)
    assert generate.generate(m, prompts, lens) == want
    assert generate.generate(m, prompts, lens, temperature=0.7, top_k=1) == want  # the sampler with one candidate
    assert m.pool_state() == (0, 8, 8)
    m.close()


def test_command_line_and_trace(tmp_path):
    vu.save_folder(tmp_path, CFG, W)
    prompt = vu.tokens(9, CFG["vocab"], 7)
    r = subprocess.run([sys.executable, "-m", "jasmine_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new", "8",
                        "--prompt", " ".join(map(str, prompt)), "--prompt", "3"], cwd=ROOT, capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr
    got = [[int(t) for t in l.split()] for l in r.stdout.strip().splitlines()]
    assert got == [greedy(CFG, W, prompt, 8), greedy(CFG, W, [3], 8)]
    toks = vu.tokens(80, CFG["vocab"], 8)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:70], "want": [69, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[70:71], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[71:], "want": [0, 8]}], "end": ["x"]}]
    for dtype in DTYPES:
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "80"],
                           input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=240)
        assert r.returncode == 0, r.stderr
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
        want = want_logits(CFG, W, toks)
        read = lambda i: np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, CFG["vocab"])
        assert vu.error(read(0), want[[69, 3]]) < TOL[dtype] and vu.error(read(2), want[[71, 79]]) < TOL[dtype]
        assert not (out / "1.f32").exists()
