"""Host side of the Vagonex design without a GPU: its configuration, the checks of sizes, and the plain implementation's own
consistency."""
import ctypes as C

import numpy as np
import pytest

import jasmine_b200 as jb
import vagonex_oracle as vo
import vagonex_util as vu
from jasmine_b200 import decoder, registry


def test_layers_come_from_the_configuration():
    layers = [vu.delta(heads=6, kv_heads=2, dim=10, vdim=14, conv=5, ff=20), vu.lightning(heads=2, dim=11, vdim=13),
              vu.attention(heads=8, kv_heads=4, dim=30, vdim=26, rot_dims=10, base=777.0, scaling=vu.YARN, size=33, scale=0.3),
              vu.attention(heads=8, kv_heads=4, dim=30, vdim=26, rot_dims=10, size=None, kv_from=2)]
    d, l, a, s = decoder.vagonex_layers(vu.config(layers))
    assert (d.mixer, d.heads, d.kv_heads, d.dim, d.vdim, d.taps, d.ff, d.ff_kind) == (jb.MIXER_DELTA, 6, 2, 10, 14, 5, 20, jb.FF_GELU_GLU)
    assert (l.mixer, l.heads, l.dim, l.vdim, l.ff) == (jb.MIXER_LINEAR_ATTENTION, 2, 11, 13, 0)
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.rot_dim, a.rope_base, a.scale) == (jb.MIXER_ATTENTION, 8, 4, 30, 26, 10, 777.0, 0.3)
    assert (a.mask, a.window, a.kv_from, a.rope_factor, a.rope_original, a.rope_fast, a.rope_slow) == (jb.MASK_CHUNK, 33, -1, 4.0, 512.0, 16.0, 2.0)
    assert (s.mask, s.kv_from, s.rope_factor) == (jb.MASK_FULL, 2, 0.0)
    assert all(k.weights_of == -1 for k in (d, l, a, s))
    bad = vu.delta()
    bad["type"] = "no such mixer"
    with pytest.raises(ValueError):
        decoder.vagonex_layers(vu.config([bad]))
    with pytest.raises(ValueError):
        decoder.vagonex_layers(vu.config([vu.lightning(heads=2, decay=[0.5])]))
    assert "Vagonex" in registry.ARCHITECTURES


def test_sizes_are_validated_before_any_device_work():
    cfg = jb.DecoderConfig(2, 16, 32, jb.F32, 2, 64, 64, 0, 1e-5, 0.0, jb.NORM_SUM, 1.0, 1.0)
    h = C.c_void_p()
    good = dict(mixer=jb.MIXER_ATTENTION, weights_of=-1, heads=4, kv_heads=2, dim=8, vdim=8, rot_dim=4, scale=1.0, rope_base=1e4, kv_from=-1,
                mask=jb.MASK_CHUNK, window=4)

    def status(second):
        arr = (jb.LayerConfig * 2)(jb.LayerConfig(**good), jb.LayerConfig(**second))
        return jb.lib().jsm_decoder_create(C.byref(cfg), arr, C.byref(h))

    for change in (dict(kv_heads=3), dict(rot_dim=3), dict(rot_dim=10), dict(window=0), dict(mask=7), dict(kv_from=1), dict(kv_from=0, heads=2), dict(kv_from=5),
                   dict(ff=-1), dict(ff_kind=9)):
        assert status({**good, **change}) == jb.INVALID_ARG, change
    rec = dict(mixer=jb.MIXER_DELTA, weights_of=-1, heads=4, kv_heads=2, dim=8, vdim=8, taps=4, kv_from=-1)
    for change in (dict(kv_heads=3), dict(taps=0), dict(dim=0)):
        assert status({**rec, **change}) == jb.INVALID_ARG, change
    assert status({**rec, "dim": 300}) == jb.UNSUPPORTED
    cfg.norm_place = 5
    assert status(good) == jb.UNSUPPORTED


def test_plain_mechanisms_agree_with_hand_written_cases():
    x = np.array([[[1.0, 2.0, 5.0, 7.0, 9.0]]])
    got = vo.rotate_interleaved(x, [3], np.array([1.0, 0.5]), 2.0)[0, 0]
    assert np.allclose(got, [2 * (np.cos(3) - 2 * np.sin(3)), 2 * (2 * np.cos(3) + np.sin(3)), 2 * (5 * np.cos(1.5) - 7 * np.sin(1.5)),
                             2 * (7 * np.cos(1.5) + 5 * np.sin(1.5)), 9.0])
    freq, mag = vo.yarn(8, 100.0, {"factor": 4.0, "original": 1000, "fast": 50.0, "slow": 1.0})
    # pair of 50 turns: 8 ln(1000 / 100 pi) / (2 ln 100) = 1.0056 -> 1; of 1 turn: 4.4033 -> 5
    assert np.allclose(freq, 100.0 ** (-np.arange(4) / 4) * (1 - 0.75 * np.array([0.0, 0.0, 0.25, 0.5]))) and np.isclose(mag, 0.1 * np.log(4) + 1)
    q = np.zeros((5, 2, 3))
    v = np.arange(5.0).reshape(5, 1, 1)
    o = vo.chunked_sink_attention(q, q[:, :1], v, 1.0, 2, [-np.inf, 0.0])
    assert np.allclose(o[:, 0, 0], [0, 0.5, 2, 2.5, 4]) and np.allclose(o[:, 1, 0], [0, 1 / 3, 1, 5 / 3, 2])
    rng = np.random.default_rng(0)
    q, k, v = (rng.standard_normal((6, 2, n)) for n in (3, 3, 4))
    for fn, extra in ((vo.decayed_sum, ([0.5, 0.9],)), (vo.delta_rule, (rng.random((6, 2)), rng.random((6, 2))))):
        part = lambda lo, hi, S: fn(q[lo:hi], k[lo:hi], v[lo:hi], *(e if isinstance(e, list) else e[lo:hi] for e in extra), S)
        y, S = part(0, 6, None)
        y1, S1 = part(0, 2, None)
        y2, S2 = part(2, 6, S1)
        assert np.allclose(np.concatenate([y1, y2]), y) and np.allclose(S, S2)
    # beta 1 and unit keys: reading a key back gives the value just written
    u = vo.unit(k)
    y, _ = vo.delta_rule(u, u, v, np.ones((6, 2)), np.ones((6, 2)))
    assert np.allclose(y, v, atol=1e-4)
    assert np.allclose(vo.causal_conv(np.array([[1.0], [2.0], [4.0]]), np.array([[10.0, 1.0]])), [[1.0], [12.0], [24.0]])
    assert np.isclose(vo.gelu_tanh(1.0), 0.8411919906)
