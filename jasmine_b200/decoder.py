"""Host-side handle of the layer-list decoder of libjasmine_b200.so (jsm_decoder_*), and the Zugolorn and Vagonex configurations.

No torch: tokens and logits are numpy arrays in host memory, the library owns the device side.  The serving calls are those
of the paged Llama handle (admit / step_active / retire / pool_state), plus open / step for portions and mixed batches."""
from __future__ import annotations

import contextlib
import ctypes as C

import numpy as np

from . import (BF16, F32, FF_GELU_GLU, MASK_CHUNK, MASK_FULL, MIXER_ATTENTION, MIXER_DELTA, MIXER_LATENT_ATTENTION, MIXER_LINEAR_ATTENTION,
               MIXER_SELECTIVE_SCAN, NORM_OUTPUT, NORM_SUM, DecoderConfig, LayerConfig, check, host_ptr, lib)


def _i32(a):
    return np.ascontiguousarray(a, dtype=np.int32)


class Decoder:
    def __init__(self, d_model, vocab, layers, norm_eps, logit_softcap=0.0, dtype="bfloat16", max_batch=8, max_context=4096,
                 max_step_tokens=2048, pool_pages=0, norm_place=NORM_OUTPUT, residual_scale=1.0, embed_scale=1.0):
        self.vocab, self.d_model, self.n_layers = vocab, d_model, len(layers)
        self.max_batch, self.max_context = max_batch, max_context
        self.stream = None  # a CUDA stream's address, or None: a stream of the model
        cfg = DecoderConfig(len(layers), d_model, vocab, {"bfloat16": BF16, "float32": F32}[dtype], max_batch, max_context,
                            max(max_step_tokens, max_batch), pool_pages, norm_eps, logit_softcap, norm_place,
                            residual_scale, embed_scale)
        self.max_step_tokens = cfg.max_step_tokens
        # most positions back that any layer looks (0: none has keys)
        self.max_window = max((max_context if k.mixer == MIXER_ATTENTION and k.mask == MASK_FULL else k.window
                               for k in layers if k.mixer in (MIXER_LATENT_ATTENTION, MIXER_ATTENTION)), default=0)
        arr = (LayerConfig * len(layers))(*layers)
        self._h = C.c_void_p()
        check(lib().jsm_decoder_create(C.byref(cfg), arr, C.byref(self._h)))

    # ---- weights ----
    def set_weight(self, name: str, array, dtype: str | None = None):
        """A tensor as a numpy array: float32, or uint16 holding bf16 bits.  Vectors and matrices."""
        a = np.ascontiguousarray(array)
        if a.dtype not in (np.float32, np.uint16):
            a = a.astype(np.float32)
        rows, cols = (a.shape[0], 1) if a.ndim == 1 else a.shape
        check(lib().jsm_decoder_set_weight(self._h, name.encode(), a.ctypes.data, F32 if a.dtype == np.float32 else BF16, rows, cols))

    def finalize(self):
        check(lib().jsm_decoder_finalize(self._h))
        return self

    # ---- serving ----
    def open(self) -> int:
        row = C.c_int()
        check(lib().jsm_decoder_seq_open(self._h, C.byref(row)))
        return row.value

    def step(self, entries, want=(), h_next=None, h_logits=None, logits=True):
        """entries: [(row, tokens)]; want: flat places among all tokens of the step.  Returns (next tokens, logits) of the
        wanted places; arrays of one's own may be passed in, logits=False leaves the logits on the device."""
        rows, counts = _i32([r for r, _ in entries]), _i32([len(t) for _, t in entries])
        ids = _i32(np.concatenate([np.asarray(t, np.int32).reshape(-1) for _, t in entries]))
        want = _i32(want)
        n = want.size
        h_next = np.empty(n, np.int32) if h_next is None else h_next
        h_logits = np.empty((n, self.vocab), np.float32) if h_logits is None and logits else h_logits
        check(lib().jsm_decoder_step(self._h, len(entries), rows.ctypes.data, counts.ctypes.data, ids.ctypes.data, n,
                                     want.ctypes.data, host_ptr(h_next), host_ptr(h_logits), self.stream))
        return h_next, h_logits

    def admit(self, h_prompt, h_logits_last=None):
        """Prefills a prompt into the next free batch row; returns (row, first generated token)."""
        if not hasattr(h_prompt, "data_ptr"):
            h_prompt = _i32(h_prompt)
        n = h_prompt.numel() if hasattr(h_prompt, "numel") else h_prompt.size
        row, tok = C.c_int(), C.c_int32()
        check(lib().jsm_decoder_seq_admit(self._h, host_ptr(h_prompt), n, C.byref(row), C.addressof(tok), host_ptr(h_logits_last), self.stream))
        return row.value, tok.value

    def step_active(self, h_ids, h_next, h_logits=None):
        check(lib().jsm_decoder_step_active(self._h, host_ptr(h_ids), host_ptr(h_next), host_ptr(h_logits), self.stream))

    def retire(self, row: int) -> int:
        """Frees the row; returns the old index of the row that moved into its place, or -1."""
        moved = C.c_int()
        check(lib().jsm_decoder_seq_retire(self._h, row, C.byref(moved), self.stream))
        return moved.value

    def pages_for(self, n_tokens: int) -> int:
        """Cache pages a sequence of n_tokens positions holds at most: pages behind every mask go back to the pool."""
        reach = min(n_tokens, self.max_window + self.max_step_tokens)
        return min(-(-n_tokens // 64), reach // 64 + 2) if self.max_window else 0

    def stream_scope(self):
        return contextlib.nullcontext()  # the library runs the model on a stream of its own

    def pool_state(self):
        a, f, t = C.c_int(), C.c_int(), C.c_int()
        check(lib().jsm_decoder_pool_state(self._h, C.byref(a), C.byref(f), C.byref(t)))
        return a.value, f.value, t.value

    def context(self, row: int) -> int:
        n = C.c_int()
        check(lib().jsm_decoder_context(self._h, row, C.byref(n)))
        return n.value

    def set_tap(self, d_buf):
        """Device buffer (a CUDA tensor, F32 [n_layers, tokens, d_model]) for the residual stream after every layer."""
        check(lib().jsm_decoder_set_tap(self._h, d_buf.data_ptr() if d_buf is not None else None))

    def step_bytes(self, context_len: int):
        w, s = C.c_uint64(), C.c_uint64()
        check(lib().jsm_decoder_step_bytes(self._h, context_len, C.byref(w), C.byref(s)))
        return w.value, s.value

    def close(self):
        if self._h:
            check(lib().jsm_decoder_destroy(self._h))
            self._h = C.c_void_p()

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass


# ---- Zugolorn ---------------------------------------------------------------------------------------------------------
def _latent_attention(mix):
    if mix["rot"]["dims"] != mix["rot_dim"]:
        raise ValueError(f"latent_attention: rot.dims {mix['rot']['dims']} differs from rot_dim {mix['rot_dim']}")
    return dict(mixer=MIXER_LATENT_ATTENTION, heads=mix["heads"], dim=mix["dim"], rot_dim=mix["rot_dim"], vdim=mix["vdim"],
                kv_rank=mix["kv_rank"], window=mix["mask"]["size"], scale=mix["scale"], rope_base=mix["rot"]["base"])


def _mamba1(mix):
    return dict(mixer=MIXER_SELECTIVE_SCAN, inner=mix["inner"], state=mix["state"], dt_rank=mix["dt_rank"], taps=mix["conv"],
                rope_base=1.0)


MIXERS = {"latent_attention": _latent_attention, "mamba1": _mamba1}


def zugolorn_layers(config: dict):
    """The layer list of a Zugolorn config.json as LayerConfig structures."""
    entries, out = config["layers"], []
    for i, e in enumerate(entries):
        if e["type"] not in MIXERS:
            raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
        kw = MIXERS[e["type"]](e["mixer"])
        mlp = e.get("mlp")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            kw.update(ff=mlp["ff"], ff_limit=mlp["limit"])
        src = i
        for _ in entries:  # a shared layer may itself share
            if entries[src].get("weights_of") is None:
                break
            src = entries[src]["weights_of"]
        out.append(LayerConfig(weights_of=-1 if src == i else src, **kw))
    return out


def zugolorn_model(config: dict, **serving) -> Decoder:
    """A Zugolorn decoder without its weights (set_weight for every tensor, then finalize)."""
    return Decoder(config["width"], config["vocab"], zugolorn_layers(config), config["norm"]["eps"],
                   config.get("logit_softcap") or 0.0, **serving)


# ---- Vagonex ----------------------------------------------------------------------------------------------------------
def _vagonex_attention(mix):
    rot, mask = mix.get("rot") or {}, mix.get("mask") or {}
    kv_from = mix.get("kv_from")
    kw = dict(mixer=MIXER_ATTENTION, heads=mix["heads"], kv_heads=mix["kv_heads"], dim=mix["dim"], vdim=mix["vdim"], scale=mix["scale"],
              rot_dim=rot.get("dims", 0), rope_base=rot.get("base", 1.0), mask=MASK_CHUNK if mask.get("size") else MASK_FULL,
              window=mask.get("size") or 0, kv_from=-1 if kv_from is None else kv_from)
    if rot.get("scaling"):
        kw.update({f"rope_{k}": float(rot["scaling"][k]) for k in ("factor", "original", "fast", "slow")})
    return kw


def _lightning(mix):
    if len(mix["decay"]) != mix["heads"]:
        raise ValueError(f"lightning: {len(mix['decay'])} decays for {mix['heads']} heads")
    return dict(mixer=MIXER_LINEAR_ATTENTION, heads=mix["heads"], dim=mix["dim"], vdim=mix["vdim"], kv_from=-1)


def _delta(mix):
    return dict(mixer=MIXER_DELTA, heads=mix["heads"], kv_heads=mix["kv_heads"], dim=mix["dim"], vdim=mix["vdim"], taps=mix["conv"], kv_from=-1)


VAGONEX_MIXERS = {"attention": _vagonex_attention, "lightning": _lightning, "delta": _delta}


def vagonex_layers(config: dict):
    """The layer list of a Vagonex config.json as LayerConfig structures."""
    out = []
    for i, e in enumerate(config["layers"]):
        if e["type"] not in VAGONEX_MIXERS:
            raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
        kw = VAGONEX_MIXERS[e["type"]](e["mixer"])
        mlp = e.get("mlp")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            kw.update(ff=mlp["ff"], ff_kind=FF_GELU_GLU)
        out.append(LayerConfig(weights_of=-1, **kw))
    return out


def vagonex_model(config: dict, **serving) -> Decoder:
    """A Vagonex decoder without its weights (set_weight for every tensor, then finalize)."""
    m = Decoder(config["width"], config["vocab"], vagonex_layers(config), config["norm"]["eps"], norm_place=NORM_SUM,
                residual_scale=config["postln_alpha"], embed_scale=config["embedding"]["scale"], **serving)
    for i, e in enumerate(config["layers"]):
        if e["type"] == "lightning":
            m.set_weight(f"l{i}.mix.decay", np.asarray(e["mixer"]["decay"], np.float32))
    return m
