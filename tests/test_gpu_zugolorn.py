"""Zugolorn on the GPU against the plain float64 implementation (zugolorn_oracle.py): each mechanism alone, prompts,
portions, decoding, batches, reuse of pages and slots, window edges, generation through the scheduler and the command line.

fp32 models are compared sharply (fp32 rounding only), bf16 models at a bf16 bar; where random weights would hide a fault,
one key is made to stand out."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import jasmine_b200 as jb
import zugolorn_oracle as zo
import zugolorn_util as zu
from gpu_util import BF16_RTOL, assert_close
from jasmine_b200 import generate, registry

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
TOL = {"float32": 4e-5, "bfloat16": 0.08}


def want_logits(cfg, w, toks):
    return zo.forward(cfg, zu.oracle_weights(w), toks)


# ---- mechanisms alone -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,N,K", [(1, 64, 64), (5, 200, 40), (16, 72, 136), (24, 328, 64), (40, 64, 520), (64, 1000, 72), (100, 136, 200), (300, 264, 96)])
def test_clamped_gate_up_projection(T, N, K):
    g = torch.Generator(device="cuda").manual_seed(T * 1000 + N)
    x = torch.randn(T, K, device="cuda", generator=g).bfloat16()
    w = (torch.randn(2 * N, K, device="cuda", generator=g) * 2 * K ** -0.5).bfloat16()
    out = torch.empty(T, N, dtype=torch.bfloat16, device="cuda")
    jb.linear_bf16_packed_glu(x, jb.linear_pack(w, N, True), out, 1.702, 0.8)
    y = x.double() @ w.double().T
    gate, up = y[:, :N].clamp(max=0.8), y[:, N:].clamp(-0.8, 0.8)
    assert_close(out.float().cpu().numpy(), (gate * torch.sigmoid(1.702 * gate) * (up + 1)).cpu().numpy(), BF16_RTOL / 2)
    jb.check_device_errors()


@pytest.mark.parametrize("T,d", [(1, 8), (3, 40), (7, 1000), (5, 2048), (4, 4096), (2, 5000)])
def test_norm_on_the_output_joins_the_residual(T, d):
    rng = np.random.default_rng(d)
    y, x, g = (rng.standard_normal(s).astype(np.float32) for s in ((T, d), (T, d), (d,)))
    want = x + zo.rms_norm(y.astype(np.float64), g.astype(np.float64), 1e-3)
    xd, xb = torch.from_numpy(x).cuda(), torch.empty(T, d, dtype=torch.bfloat16, device="cuda")
    jb.post_norm_add(torch.from_numpy(y).cuda(), xd, torch.from_numpy(g).cuda(), 1e-3, xb)
    assert_close(xd.cpu().numpy(), want, 1e-6)
    assert torch.equal(xb, xd.bfloat16())


@pytest.mark.parametrize("vocab,pitch,cap", [(5, 8, 2.0), (72, 72, 5.0), (5003, 5008, 3.0), (40000, 40000, 0.0)])
def test_capped_logits_and_their_maximum(vocab, pitch, cap):
    rng = np.random.default_rng(vocab)
    x = (4 * rng.standard_normal((3, pitch))).astype(np.float32)
    x[1, vocab // 2] = x[1, vocab // 3] = 30.0  # a tie: the first wins, also after the cap saturates
    t = torch.from_numpy(x.copy()).cuda()
    nxt = jb.logits_finish(t, vocab, cap)
    want = zo.softcap(x.astype(np.float64), cap) if cap else x
    got = t.cpu().numpy()
    assert_close(got[:, :vocab], want[:, :vocab], 1e-6)
    assert np.array_equal(got[:, vocab:], x[:, vocab:])
    assert nxt.tolist() == np.argmax(got[:, :vocab], axis=1).tolist() and nxt[1] == vocab // 3


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


ATTENTION = [dict(), dict(heads=1, dim=8, rot_dim=2, vdim=8, kv_rank=8, window=1), dict(heads=5, dim=9, rot_dim=6, vdim=13, kv_rank=17, window=7),
             dict(heads=2, dim=33, rot_dim=10, vdim=40, kv_rank=70, window=64), dict(heads=7, dim=24, rot_dim=40, vdim=24, kv_rank=130, window=65, base=300.0, scale=0.31),
             dict(heads=4, dim=48, rot_dim=16, vdim=64, kv_rank=272, window=128), dict(heads=33, dim=16, rot_dim=16, vdim=8, kv_rank=24, window=100),
             dict(heads=2, dim=64, rot_dim=64, vdim=96, kv_rank=400, window=90), dict(heads=2, dim=130, rot_dim=30, vdim=128, kv_rank=64, window=500),
             dict(heads=2, dim=200, rot_dim=32, vdim=140, kv_rank=530, window=70), dict(heads=2, dim=24, rot_dim=136, vdim=16, kv_rank=140, window=80)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kw", ATTENTION, ids=lambda k: "-".join(map(str, k.values())) or "default")
def test_latent_attention_alone(kw, dtype):
    cfg = zu.config([zu.attention(**kw)], width=56)
    w = zu.random_weights(cfg, 3)
    toks = zu.tokens(150, cfg["vocab"], 4)
    want = []
    zo.forward(cfg, zu.oracle_weights(w), toks, want)
    m = zu.build(cfg, w, dtype)
    for sizes in ([150], [70, 2, 50, 28], [1] * 20 + [97] + [1] * 33):
        assert_close(layer_residual(m, toks, sizes)[0], want[0], 1e-5 if dtype == "float32" else BF16_RTOL, str(sizes[:3]))
    m.close()


SCAN = [dict(), dict(inner=8, state=1, dt_rank=1, conv=1), dict(inner=33, state=7, dt_rank=9, conv=2), dict(inner=100, state=16, dt_rank=20, conv=3),
        dict(inner=64, state=24, dt_rank=4, conv=5), dict(inner=20, state=33, dt_rank=2, conv=4), dict(inner=70, state=100, dt_rank=37, conv=6)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kw", SCAN, ids=lambda k: "-".join(map(str, k.values())) or "default")
def test_selective_scan_alone(kw, dtype):
    cfg = zu.config([zu.mamba(**kw)])
    w = zu.random_weights(cfg, 5)
    toks = zu.tokens(140, cfg["vocab"], 6)
    want = []
    zo.forward(cfg, zu.oracle_weights(w), toks, want)
    m = zu.build(cfg, w, dtype)
    for sizes in ([140], [2, 3, 31, 1, 1, 64, 38], [1] * 40 + [100]):
        assert_close(layer_residual(m, toks, sizes)[0], want[0], 1e-5 if dtype == "float32" else BF16_RTOL, str(sizes[:3]))
    m.close()


def test_scan_state_decays_slowly_enough_to_matter():
    """Slow decays: the first token's trace survives hundreds of steps, so a state lost anywhere shows."""
    cfg = zu.config([zu.mamba(inner=32, state=4)])
    w = zu.random_weights(cfg, 7)
    w["l0.mix.A_log"] = zu.bf16_bits(np.full((32, 4), -6.0))
    toks = zu.tokens(400, cfg["vocab"], 8)
    other = [(toks[0] + 1) % cfg["vocab"]] + toks[1:]
    want = want_logits(cfg, w, toks)
    assert zu.error(want_logits(cfg, w, other)[-1:], want[-1:]) > 100 * TOL["float32"]
    m = zu.build(cfg, w)
    for sizes in ([400], [150, 2, 1, 200], [3]):
        assert zu.error(zu.run_portions(m, toks, sizes)[-1:], want[-1:]) < TOL["float32"]
    m.close()


# ---- whole models -----------------------------------------------------------------------------------------------------
def mixed_config():
    layers = [zu.mamba(inner=56, state=6, dt_rank=5, conv=3, ff=88, limit=0.9), zu.attention(heads=3, window=50),
              zu.attention(heads=5, dim=24, rot_dim=12, vdim=20, kv_rank=40, window=90, base=500.0, ff=100, limit=1.2),
              zu.mamba(inner=40, state=16, dt_rank=2, conv=4)]
    layers += [zu.shared(layers, 2), zu.shared(layers, 0), zu.attention(heads=2, window=33, ff=24)]
    return zu.config(layers, width=52, vocab=101)


CFG = mixed_config()
W = zu.random_weights(CFG, 11)


@pytest.fixture(scope="module", params=["float32", "bfloat16"])
def model(request):
    m = zu.build(CFG, W, request.param, max_batch=6)
    m.dtype_name = request.param
    yield m
    m.close()


@pytest.fixture(scope="module")
def long_case():
    toks = zu.tokens(330, CFG["vocab"], 12)
    return toks, want_logits(CFG, W, toks)


@pytest.mark.parametrize("sizes", [[330], [1], [2], [3, 5, 7], [64], [63, 65], [130, 1, 1, 140], [200, 2], [33, 50, 90]], ids=str)
def test_portions_of_a_prompt(model, long_case, sizes):
    toks, want = long_case
    assert zu.error(zu.run_portions(model, toks, sizes), want) < TOL[model.dtype_name]


def test_first_tokens(model):
    for n in (1, 2, 3, 4, 5):
        toks = zu.tokens(n, CFG["vocab"], 40 + n)
        want = want_logits(CFG, W, toks)
        for sizes in ([n], [1]):
            assert zu.error(zu.run_portions(model, toks, sizes), want) < TOL[model.dtype_name]


def test_batches_of_unequal_requests(model):
    """Prompts, portions and single tokens of several sequences in one step: each as if it were alone."""
    tol = TOL[model.dtype_name]
    seqs = [zu.tokens(n, CFG["vocab"], 60 + n) for n in (260, 17, 140, 1, 75)]
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
            assert zu.error(lg[k:k + 1], want[i][p:p + 1]) < tol, (i, p)
            assert nxt[k] == int(np.argmax(lg[k]))
    for _ in rows:
        model.retire(0)
    assert model.pool_state()[0] == 0


def test_pages_and_slots_are_used_again():
    """A pool too small for all sequences at once, rows that move, windows that give pages back while a sequence runs."""
    m = zu.build(CFG, W, "float32", max_batch=3, max_context=512, max_step_tokens=96, pool_pages=10)
    seqs = {k: zu.tokens(n, CFG["vocab"], 80 + k) for k, n in enumerate((400, 90, 200, 30, 150))}
    want = {k: want_logits(CFG, W, s) for k, s in seqs.items()}
    rows, at, todo = [], {}, [0, 1, 2, 3, 4]

    def advance(k, n):
        n = min(n, len(seqs[k]) - at[k])
        _, lg = m.step([(rows.index(k), seqs[k][at[k]:at[k] + n])], range(n))
        assert zu.error(lg, want[k][at[k]:at[k] + n]) < TOL["float32"], (k, at[k])
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
    assert m.pool_state() == (0, 10, 10)  # every page is back
    with pytest.raises(jb.JsmError) as e:
        for _ in range(4):
            m.open()
    assert e.value.status == jb.OOM
    m.close()


def test_a_refused_admission_takes_nothing():
    cfg = zu.config([zu.attention(window=400)])
    m = zu.build(cfg, zu.random_weights(cfg, 1), max_batch=2, max_context=512, pool_pages=3)
    row, _ = m.admit(np.arange(100) % 72)
    assert m.pool_state() == (1, 1, 3)
    with pytest.raises(jb.JsmError) as e:
        m.admit(np.arange(150) % 72)
    assert e.value.status == jb.OOM and m.pool_state() == (1, 1, 3)
    with pytest.raises(jb.JsmError) as e:
        m.step([(0, [1000])])
    assert e.value.status == jb.INVALID_ARG
    m.retire(row)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 100, 128, 129])
def test_edges_of_a_window(window, dtype):
    """One key stands out: token 0 of the vocabulary attracts every query.  It is placed so that a query sees it as the
    last key of its window, and the next query does not any more; in prompts (short and long) and in decoding."""
    cfg = zu.config([zu.attention(heads=2, dim=16, rot_dim=2, vdim=16, kv_rank=16, window=window, scale=1.0)], width=48)
    w = zu.random_weights(cfg, 21)
    d = 48
    rng = np.random.default_rng(5)
    emb = zu.widen(w["embed"]).reshape(-1, d)
    emb[:, 0], emb[:, 1] = 1.0, 0.0
    emb[0] = 0.0
    emb[0, 1] = 6.0                       # the key token
    q = np.zeros((2 * 18, d))
    q[[0, 18], 0] = 12.0                  # every other token asks for component 0 of the key
    dkv = 0.3 * rng.standard_normal((18, d))
    dkv[0] = 0.0
    dkv[0, 1] = 4.0                       # which only the key token has
    uk = np.zeros((32, 16))
    uk[[0, 16], 0] = 1.0
    w.update({"embed": zu.bf16_bits(emb), "l0.mix.q": zu.bf16_bits(q), "l0.mix.dkv": zu.bf16_bits(dkv), "l0.mix.uk": zu.bf16_bits(uk)})
    m = zu.build(cfg, w, dtype)
    tol = TOL[dtype]
    for place in (0, 1, 62, 64):
        toks = [1 + t % 71 for t in zu.tokens(place + window + 140, 71, 30 + place)]
        toks[place] = 0
        want = want_logits(cfg, w, toks)
        inside, outside = place + window - 1, place + window
        wider = json.loads(json.dumps(cfg))
        wider["layers"][0]["mixer"]["mask"]["size"] = window + 1
        assert zu.error(want_logits(wider, w, toks)[outside:outside + 1], want[outside:outside + 1]) > 3 * TOL["bfloat16"]  # the edge shows
        for sizes in ([len(toks)], [max(1, inside - 1), 2], [inside + 1, 1], [1] * 3 + [max(1, inside)] + [1], [130, 1]):
            got = zu.run_portions(m, toks, sizes)
            assert zu.error(got[inside:outside + 2], want[inside:outside + 2]) < tol, (place, sizes[:3])
            assert zu.error(got, want) < tol
    m.close()


FLASH = [dict(heads=2, dim=40, rot_dim=24, vdim=64), dict(heads=3, dim=48, rot_dim=16, vdim=100), dict(heads=2, dim=70, rot_dim=30, vdim=30),
         dict(heads=2, dim=96, rot_dim=32, vdim=128), dict(heads=3, dim=100, rot_dim=60, vdim=60), dict(heads=2, dim=128, rot_dim=64, vdim=128)]


@pytest.mark.parametrize("window", [20, 128, 200, 257, 2000])
@pytest.mark.parametrize("kw", FLASH, ids=lambda k: "-".join(map(str, k.values())))
def test_long_prompts_take_the_flash_kernel(kw, window):
    """Segments of at least 128 tokens expand keys and values; every tile shape, windows shorter and longer than a tile,
    portions that start inside a page and a tile."""
    cfg = zu.config([zu.attention(kv_rank=48, window=window, **kw)], width=64)
    w = zu.random_weights(cfg, 31, q_gain=3.0)
    toks = zu.tokens(700, cfg["vocab"], 32)
    want = []
    zo.forward(cfg, zu.oracle_weights(w), toks, want)
    m = zu.build(cfg, w, "bfloat16")
    for sizes in ([700], [129, 300, 271], [37, 400, 3, 260], [690] + [1] * 10):
        got = layer_residual(m, toks, sizes)[0]
        assert_close(got, want[0], 1.5 * BF16_RTOL, str(sizes))
        assert zu.error(got, want[0]) < 0.02
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_kind_of_mixer_only(dtype):
    """Models without attention (no pages) and without recurrence (no states)."""
    for layers in ([zu.mamba(ff=24), zu.mamba(inner=24)], [zu.attention(ff=24), zu.attention(window=9)]):
        cfg = zu.config(layers)
        w = zu.random_weights(cfg, 51)
        m = zu.build(cfg, w, dtype, max_batch=2, max_context=100)
        for seed in (52, 53):
            toks = zu.tokens(90, cfg["vocab"], seed)
            assert zu.error(zu.run_portions(m, toks, [60, 2, 1]), want_logits(cfg, w, toks)) < TOL[dtype]
        assert generate.generate(m, [toks[:5], toks[:30]], 4)[0]
        m.close()


def test_steps_longer_than_a_pass_are_cut():
    m = zu.build(CFG, W, "float32", max_step_tokens=50)
    toks = zu.tokens(233, CFG["vocab"], 90)
    assert zu.error(zu.run_portions(m, toks, [233]), want_logits(CFG, W, toks)) < TOL["float32"]
    m.close()


def test_long_decoding(model):
    toks = zu.tokens(420, CFG["vocab"], 91)
    want = want_logits(CFG, W, toks)
    got = zu.run_portions(model, toks, [20, 1])  # far past every window
    assert zu.error(got, want) < TOL[model.dtype_name]


# ---- generation -------------------------------------------------------------------------------------------------------
def greedy(cfg, w, prompt, n):
    seq = list(prompt)
    ow = zu.oracle_weights(w)
    for _ in range(n):
        seq.append(int(np.argmax(zo.forward(cfg, ow, seq)[-1])))
    return seq[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    prompts = [zu.tokens(n, CFG["vocab"], 100 + n) for n in (5, 70, 1, 33, 18)]
    lens = [12, 6, 15, 3, 9]
    want = [greedy(CFG, W, p, n) for p, n in zip(prompts, lens)]
    m = zu.build(CFG, W, "float32", max_batch=3, max_context=128, pool_pages=8)
    assert generate.generate(m, prompts, lens) == want
    assert generate.generate(m, prompts, lens, temperature=0.7, top_k=1) == want  # the sampler with one candidate
    a = generate.generate(m, prompts, lens, temperature=1.0, seed=1)
    assert a == generate.generate(m, prompts, lens, temperature=1.0, seed=1) and a != want
    assert m.pool_state() == (0, 8, 8)
    m.close()


def test_command_line_and_trace(tmp_path):
    zu.save_folder(tmp_path, CFG, W)
    prompt = zu.tokens(9, CFG["vocab"], 7)
    r = subprocess.run([sys.executable, "-m", "jasmine_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new", "8",
                        "--prompt", " ".join(map(str, prompt)), "--prompt", "3"], cwd=ROOT, capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr
    got = [[int(t) for t in l.split()] for l in r.stdout.strip().splitlines()]
    assert got == [greedy(CFG, W, prompt, 8), greedy(CFG, W, [3], 8)]
    toks = zu.tokens(80, CFG["vocab"], 8)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:70], "want": [69, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[70:71], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[71:], "want": [0, 8]}], "end": ["x"]}]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "80"],
                           input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=240)
        assert r.returncode == 0, r.stderr
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
        want = want_logits(CFG, W, toks)
        read = lambda i: np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, CFG["vocab"])
        assert zu.error(read(0), want[[69, 3]]) < TOL[dtype] and zu.error(read(2), want[[71, 79]]) < TOL[dtype]
        assert not (out / "1.f32").exists()


def test_llama_is_served_by_the_same_scheduler(tmp_path):
    cfg = {"architecture": "Llama", "n_layers": 2, "d_model": 256, "n_heads": 2, "n_kv_heads": 2, "d_ffn": 512, "vocab": 1024, "seed": 4}
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    prompts = [zu.tokens(n, 1024, n) for n in (12, 80, 5)]
    m = registry.load_model(tmp_path, max_batch=2, max_context=128, pool_pages=4)
    got = generate.generate(m, prompts, 6)
    alone = [generate.generate(m, [p], 6)[0] for p in prompts]
    assert all(len(g) == 6 for g in got) and [g[0] for g in got] == [a[0] for a in alone]
    assert m.pool_state() == (0, 4, 4)
    m.close()
