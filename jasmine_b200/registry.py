"""Model registry: a folder with config.json -> a model ready to serve.

config.json names its design under "architecture"; every design registers a loader.  All models serve the same calls
(admit / step_active / retire / pool_state), which is what generate.py schedules."""
from __future__ import annotations

import json
from pathlib import Path

from . import JsmError, UNSUPPORTED
from .safetensors import SafeTensors

ARCHITECTURES = {}


def register(name):
    def add(fn):
        ARCHITECTURES[name] = fn
        return fn
    return add


def read_config(folder) -> dict:
    return json.loads((Path(folder) / "config.json").read_text())


def load_model(folder, dtype="bfloat16", **serving):
    """serving: max_batch, max_context, max_step_tokens, pool_pages (what a design does not have, it ignores)."""
    config = read_config(folder)
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise JsmError(UNSUPPORTED, f"unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    return ARCHITECTURES[name](Path(folder), config, dtype, serving)


def _layer_list(make, folder, config, dtype, serving):
    """A layer-list decoder (decoder.py) with the tensors of model.safetensors."""
    model = make(config, dtype=dtype, **serving)
    weights = SafeTensors(folder / "model.safetensors")
    for name in weights:
        kind, array = weights.get(name)
        if kind not in ("BF16", "F32"):
            raise JsmError(UNSUPPORTED, f"tensor {name}: dtype {kind}")
        model.set_weight(name, array)
    return model.finalize()


@register("Zugolorn")
def _zugolorn(folder, config, dtype, serving):
    from .decoder import zugolorn_model
    return _layer_list(zugolorn_model, folder, config, dtype, serving)


@register("Vagonex")
def _vagonex(folder, config, dtype, serving):
    from .decoder import vagonex_model
    return _layer_list(vagonex_model, folder, config, dtype, serving)


@register("Llama")
def _llama(folder, config, dtype, serving):
    """LLaMA-shape decoder: config.json holds the sizes, model.jsm the checkpoint that Llama.save wrote (without one, the
    weights are generated from "seed")."""
    from .model import Llama
    if dtype != "bfloat16":
        raise JsmError(UNSUPPORTED, f"Llama runs in bfloat16 only ({dtype} asked for)")
    max_batch, max_context = serving.get("max_batch", 8), serving.get("max_context", 4096)
    pages = serving.get("pool_pages") or max_batch * -(-max_context // 64)
    model = Llama(config["n_layers"], config["d_model"], config["n_heads"], config["n_kv_heads"], config["d_ffn"], config["vocab"],
                  max_batch, max_context, config.get("head_dim", 128), config.get("norm_eps", 1e-5),
                  config.get("rope_theta", 10000.0), config.get("seed", 4), pool_pages=pages)
    if (folder / "model.jsm").exists():
        model.load(folder / "model.jsm")
    return model
