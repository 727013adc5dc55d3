"""Model registry: which class serves a folder with config.json and model.safetensors, and how it is loaded.

`load(dev, folder)` picks the entry by config.json ("architecture", or Hugging Face's "architectures" / "model_type").
Quantized models (Llama, GPT-2) take `bits` and `group` unless the file holds quantized weights already; `dtype` is the
number format of the models that run unquantized (Zazasun, Lotorax).
"""
import json
import os

from . import checkpoint, nn

DTYPES = ("bfloat16", "float32")


def _llama_config(c):
    heads, d = c["num_attention_heads"], c["hidden_size"]
    return nn.LlamaConfig(c["vocab_size"], d, c["intermediate_size"], c["num_hidden_layers"], heads, c.get("num_key_value_heads") or heads,
                          c.get("head_dim") or d // heads, c["max_position_embeddings"], c.get("rms_norm_eps", 1e-5), c.get("rope_theta", 10000.0),
                          int(c.get("tie_word_embeddings", False)))


def _gpt2_config(c):
    return nn.GPT2Config(c["vocab_size"], c["n_positions"], c["n_embd"], c["n_layer"], c["n_head"])


def _load_llama(dev, c, path, dtype, bits, group):
    return checkpoint.load_llama(dev, _llama_config(c), path, bits, group)


def _load_gpt2(dev, c, path, dtype, bits, group):
    return checkpoint.load_gpt2(dev, _gpt2_config(c), path, bits, group)


def _load_zazasun(dev, c, path, dtype, bits, group):
    if bits is not None:
        raise ValueError("Zazasun runs unquantized: choose a dtype, not bits")
    return checkpoint.load_zazasun(dev, c, path, dtype)


def _load_lotorax(dev, c, path, dtype, bits, group):
    if bits is not None:
        raise ValueError("Lotorax runs unquantized: choose a dtype, not bits")
    return checkpoint.load_lotorax(dev, c, path, dtype)


MODELS = {"llama": _load_llama, "gpt2": _load_gpt2, "zazasun": _load_zazasun, "lotorax": _load_lotorax}
_ALIASES = {"llamaforcausallm": "llama", "gpt2lmheadmodel": "gpt2"}


def architecture(config):
    """Registry name of a config.json's model."""
    for name in [config.get("architecture"), *(config.get("architectures") or []), config.get("model_type")]:
        if name:
            key = str(name).lower()
            key = _ALIASES.get(key, key)
            if key in MODELS:
                return key
    raise ValueError(f"no model for this configuration; known: {', '.join(sorted(MODELS))}")


def read_config(folder):
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def load(dev, folder, dtype="bfloat16", bits=None, group=32):
    if dtype not in DTYPES:
        raise ValueError(f"dtype {dtype!r}: one of {', '.join(DTYPES)}")
    config = read_config(folder)
    return MODELS[architecture(config)](dev, config, os.path.join(folder, "model.safetensors"), dtype, bits, group)
