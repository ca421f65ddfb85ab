"""Host logic of the layer-list decoder and of serving, without a GPU: configuration, weight files, registry, trace replay,
the scheduler (with a fake model), and the plain implementation's own consistency."""
import ctypes as C
import json

import numpy as np
import pytest

import jasmine_b200 as jb
import zugolorn_oracle as zo
import zugolorn_util as zu
from jasmine_b200 import decoder, generate, registry, trace
from jasmine_b200.safetensors import SafeTensors


def test_layers_come_from_the_configuration():
    layers = [zu.attention(heads=5, dim=10, rot_dim=4, vdim=7, kv_rank=9, window=33, base=777.0, scale=0.3, ff=20, limit=0.7),
              zu.mamba(inner=11, state=3, dt_rank=2, conv=5)]
    layers += [zu.shared(layers, 0), zu.shared(layers, 1)]
    chain = zu.shared(layers, 0)
    chain["weights_of"] = 2
    got = decoder.zugolorn_layers(zu.config(layers + [chain]))
    a, s = got[0], got[1]
    assert (a.mixer, a.weights_of, a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.window) == (0, -1, 5, 10, 4, 7, 9, 33)
    assert (a.ff, a.scale, a.rope_base) == (20, 0.3, 777.0) and abs(a.ff_limit - 0.7) < 1e-7
    assert (s.mixer, s.weights_of, s.inner, s.state, s.dt_rank, s.taps, s.ff) == (1, -1, 11, 3, 2, 5, 0)
    assert [g.weights_of for g in got] == [-1, -1, 0, 1, 0]
    bad = zu.attention()
    bad["type"] = "no such mixer"
    with pytest.raises(ValueError):
        decoder.zugolorn_layers(zu.config([bad]))


def test_sizes_are_validated_before_any_device_work():
    cfg = jb.DecoderConfig(1, 16, 32, jb.F32, 2, 64, 64, 0, 1e-5, 0.0)
    h = C.c_void_p()
    bad = (jb.LayerConfig * 1)(jb.LayerConfig(mixer=0, weights_of=-1, heads=2, dim=8, rot_dim=3, vdim=8, kv_rank=8, window=4, scale=1.0, rope_base=1e4))
    assert jb.lib().jsm_decoder_create(C.byref(cfg), bad, C.byref(h)) == jb.INVALID_ARG  # odd rotated part
    bad[0] = jb.LayerConfig(mixer=1, weights_of=-1, inner=8, state=200, dt_rank=1, taps=4, rope_base=1.0)
    assert jb.lib().jsm_decoder_create(C.byref(cfg), bad, C.byref(h)) == jb.UNSUPPORTED
    bad[0] = jb.LayerConfig(mixer=1, weights_of=0, inner=8, state=2, dt_rank=1, taps=4, rope_base=1.0)
    assert jb.lib().jsm_decoder_create(C.byref(cfg), bad, C.byref(h)) == jb.INVALID_ARG  # its own weights


def test_safetensors_round_trip(tmp_path):
    cfg = zu.config([zu.mamba()])
    w = zu.random_weights(cfg, 1)
    zu.save_folder(tmp_path, cfg, w)
    st = SafeTensors(tmp_path / "model.safetensors")
    assert set(st) == set(w)
    for k, v in w.items():
        kind, a = st.get(k)
        assert kind == "BF16" and np.array_equal(a, v)
    assert registry.read_config(tmp_path) == json.loads(json.dumps(cfg))


def test_registry_names_unknown_designs(tmp_path):
    (tmp_path / "config.json").write_text('{"architecture": "Nobody"}')
    with pytest.raises(jb.JsmError) as e:
        registry.load_model(tmp_path)
    assert e.value.status == jb.UNSUPPORTED and "Zugolorn" in str(e.value)
    (tmp_path / "config.json").write_text('{"architecture": "Llama"}')
    with pytest.raises(jb.JsmError):
        registry.load_model(tmp_path, "float32")


class FakeModel:
    """The serving calls of a model whose next token is (sum of the sequence) % vocab; checks the row discipline."""
    vocab, max_context = 97, 64

    def __init__(self, max_batch, pages):
        self.max_batch, self.pages, self.rows, self.peak = max_batch, pages, [], 0

    def pages_for(self, n):
        return -(-n // 8)

    def pool_state(self):
        used = sum(self.pages_for(len(r)) for r in self.rows)
        return len(self.rows), self.pages - used, self.pages

    def stream_scope(self):
        import contextlib
        return contextlib.nullcontext()

    def open(self):
        assert len(self.rows) < self.max_batch
        self.rows.append([])
        return len(self.rows) - 1

    def admit(self, prompt, logits=None):
        row = self.open()
        self.rows[row] = [int(t) for t in prompt]
        assert self.pool_state()[1] >= 0
        return row, sum(self.rows[row]) % self.vocab

    def step_active(self, ids, nxt, logits=None):
        self.peak = max(self.peak, len(self.rows))
        for i, r in enumerate(self.rows):
            r.append(int(ids[i]))
            nxt[i] = sum(r) % self.vocab
        assert self.pool_state()[1] >= 0, "the scheduler over-committed the pages"

    def step(self, entries, want):
        flat = []
        for row, toks in entries:
            for t in toks:
                self.rows[row].append(int(t))
                flat.append(sum(self.rows[row]))
        return None, np.asarray([[flat[w]] * 2 for w in want], np.float32)

    def retire(self, row):
        last = self.rows.pop()
        if row == len(self.rows):
            return -1
        self.rows[row] = last
        return len(self.rows)


def test_scheduler_serves_every_prompt_within_rows_and_pages():
    prompts = [zu.tokens(n, 97, 10 + n) for n in (3, 20, 1, 9, 33, 14, 2)]
    lens = [5, 1, 12, 7, 20, 3, 0]
    m = FakeModel(3, 9)
    got = generate.generate(m, prompts, lens)
    assert m.rows == [] and m.peak <= 3
    for p, n, g in zip(prompts, lens, got):
        want, seq = [], list(p)
        for _ in range(n):
            want.append(sum(seq) % 97)
            seq.append(want[-1])
        assert g == want
    first = got[0][2]
    assert generate.generate(FakeModel(2, 20), prompts[:1], 5, stop=[first])[0] == got[0][:got[0].index(first) + 1]
    with pytest.raises(jb.JsmError):
        generate.generate(FakeModel(2, 20), [[1] * 60], 5)
    with pytest.raises(jb.JsmError):
        generate.generate(FakeModel(2, 2), [[1] * 20], 5)


def test_trace_replay_follows_rows_that_move(tmp_path):
    m = FakeModel(4, 100)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2], "want": [1, 0]}, {"id": "b", "tokens": [5], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "c", "tokens": [7, 7, 7], "want": [2]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "c", "tokens": [1], "want": [0]}, {"id": "b", "tokens": [10], "want": [0]}], "end": ["b", "c"]},
             {"step": 3, "entries": [{"id": "a", "tokens": [9], "want": []}], "end": ["a"]}]
    told = []
    trace.replay(m, [json.dumps(s) for s in steps], tmp_path, told.append)
    assert told == [f"done {i}" for i in range(4)] and m.rows == []
    read = lambda i: np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, 2)[:, 0].tolist()
    assert read(0) == [3, 1] and read(1) == [21] and read(2) == [22, 15]
    assert not (tmp_path / "3.f32").exists()


def test_plain_mechanisms_agree_with_hand_written_cases():
    assert np.allclose(zo.rotate_half(np.array([[1.0, 0.0, 2.0, 0.0]]), [3], 100.0),
                       [[np.cos(3) - 2 * np.sin(3), 0, 2 * np.cos(3) + np.sin(3), 0]])
    x = np.array([[1.0], [2.0], [4.0]])
    assert np.allclose(zo.causal_conv(x, np.array([[10.0, 1.0]]), np.array([0.5])), [[1.5], [12.5], [24.5]])
    rng = np.random.default_rng(0)
    a = [rng.standard_normal(s) for s in ((6, 3), (6, 3), (3, 2), (6, 2), (6, 2), (3,))]
    a[1] = np.abs(a[1])
    y, S = zo.selective_scan(*a)
    y1, S1 = zo.selective_scan(a[0][:4], a[1][:4], a[2], a[3][:4], a[4][:4], a[5])
    y2, S2 = zo.selective_scan(a[0][4:], a[1][4:], a[2], a[3][4:], a[4][4:], a[5], S1)
    assert np.allclose(np.concatenate([y1, y2]), y) and np.allclose(S, S2)
    q = rng.standard_normal((5, 1, 2))
    o = zo.window_softmax_attention(q, q, q, 1.0, 1)
    assert np.allclose(o, q)  # a window of one sees itself only
    assert np.allclose(zo.clamped_glu(np.array([[2.0]]), {"gate": np.array([[5.0]]), "up": np.array([[-5.0]]), "down": np.array([[1.0]])}, 3.0),
                       3 * zo.sigmoid(1.702 * 3) * -2)
