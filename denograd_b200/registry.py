"""Models by configuration: a folder with config.json and weights -> the driver that serves it."""
from __future__ import annotations

import json
import os

class UnsupportedDtype(ValueError):
    pass


def _weights_path(folder: str) -> str:
    for name in ("model.safetensors.index.json", "model.safetensors"):
        if os.path.exists(os.path.join(folder, name)):
            return os.path.join(folder, name)
    raise FileNotFoundError(f"{folder}: no model.safetensors")


def _hybrid(config: dict, folder: str, dtype: str | None, max_context: int, max_batch: int, **kw):
    from . import build, ffi
    ffi.use_component(build.component_of(lc["type"] for lc in config["layers"]))
    from .matulorn import Matulorn
    from .rigazen import Rigazen
    cls = {c.architecture: c for c in (Matulorn, Rigazen)}[architecture(config)]
    return cls(config, dtype or "bfloat16", max_context, max_batch, **kw).load_weights(_weights_path(folder))


def _llama(config: dict, folder: str, dtype: str | None, max_context: int, max_batch: int, **kw):
    if dtype not in (None, "float16", "int8", "nf4", "bfloat16"):
        raise UnsupportedDtype(f"Llama runs with float16 activations; dtype {dtype!r} is not available")
    from .llama3 import Llama3
    args = {"dim": config["hidden_size"], "n_heads": config["num_attention_heads"], "n_layers": config["num_hidden_layers"],
            "n_kv_heads": config.get("num_key_value_heads", config["num_attention_heads"]), "norm_eps": config["rms_norm_eps"],
            "rope_theta": config.get("rope_theta", 10000.0), "vocab_size": config["vocab_size"], "hidden_dim": config["intermediate_size"]}
    quant = dtype if dtype in ("int8", "nf4") else "float16"
    return Llama3(size="8B", args=args, quantize=quant, max_context=max_context, max_batch=max_batch,
                  tied_output=bool(config.get("tie_word_embeddings", False)), **kw).load_weights(_weights_path(folder))


# architecture name in config.json -> loader
ARCHITECTURES = {"Matulorn": _hybrid, "Rigazen": _hybrid, "LlamaForCausalLM": _llama}


def architecture(config: dict) -> str:
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    if name not in ARCHITECTURES:
        raise ValueError(f"architecture {name!r} is not known (known: {', '.join(ARCHITECTURES)})")
    return name


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def load(folder: str, dtype: str | None = None, max_context: int = 8192, max_batch: int = 1, **kw):
    """The driver of the model in `folder`, weights loaded.  dtype None: the one the model is served with."""
    config = read_config(folder)
    return ARCHITECTURES[architecture(config)](config, folder, dtype, max_context, max_batch, **kw)
