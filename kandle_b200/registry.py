"""Model registry: a checkpoint folder's config.json names its architecture, the architecture names the
configuration and the engine."""
from __future__ import annotations

import json
import os

from . import io

_MODELS: dict = {}


class ModelEntry:
    """config: config.json dict, dtype -> configuration; engine: (configuration, weights, max_batch, max_seq_len) -> engine."""

    def __init__(self, config, engine, dtypes):
        self.config, self.engine, self.dtypes = config, engine, tuple(dtypes)


def register(name: str, entry: ModelEntry) -> None:
    _MODELS[name] = entry


def architectures() -> list:
    return sorted(_MODELS)


def lookup(config: dict) -> ModelEntry:
    names = [config["architecture"]] if "architecture" in config else list(config.get("architectures") or [])
    for n in names:
        if n in _MODELS:
            return _MODELS[n]
    raise ValueError(f"config.json names {names or 'no architecture'}; known: {architectures()}")


def load_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json"), encoding="utf-8") as f:
        return json.load(f)


def load_engine(folder: str, max_batch: int, max_seq_len: int, dtype: str = "bfloat16"):
    """Engine with the weights of `folder` (config.json and model.safetensors, or an index of shards)."""
    config = load_config(folder)
    entry = lookup(config)
    if dtype not in entry.dtypes:
        raise ValueError(f"dtype {dtype!r}: this architecture runs in {', '.join(entry.dtypes)}")
    index = os.path.join(folder, "model.safetensors.index.json")
    group = io.loadSafetensor(index if os.path.exists(index) else os.path.join(folder, "model.safetensors"))
    try:
        return entry.engine(entry.config(config, dtype), io.SafetensorStateDict(group), max_batch, max_seq_len)
    finally:
        group.close()


def _qwen3_config(c: dict, dtype: str):
    from .model_utils.qwen3 import Qwen3Config
    return Qwen3Config(vocabSize=c["vocab_size"], hiddenSize=c["hidden_size"], intermediateSize=c["intermediate_size"],
                       numHiddenLayers=c["num_hidden_layers"], numAttentionHeads=c["num_attention_heads"],
                       numKeyValueHeads=c["num_key_value_heads"], headDim=c.get("head_dim", c["hidden_size"] // c["num_attention_heads"]),
                       rmsNormEps=c.get("rms_norm_eps", 1e-6), ropeTheta=c.get("rope_theta", 1e6), dtype=dtype)


def _qwen3_engine(cfg, weights, max_batch, max_seq_len):
    from .engine import Qwen3Engine
    return Qwen3Engine(cfg, weights, max_batch, max_seq_len)


def _pedorax_config(c: dict, dtype: str):
    from .model_utils.pedorax import PedoraxConfig
    return PedoraxConfig.fromDict(c, dtype)


def _vogozen_config(c: dict, dtype: str):
    from .model_utils.vogozen import VogozenConfig
    return VogozenConfig.fromDict(c, dtype)


def _hybrid_engine(cfg, weights, max_batch, max_seq_len):
    from .hybrid_engine import HybridEngine
    return HybridEngine(cfg, weights, max_batch, max_seq_len)


register("Qwen3ForCausalLM", ModelEntry(_qwen3_config, _qwen3_engine, ("bfloat16",)))
register("Pedorax", ModelEntry(_pedorax_config, _hybrid_engine, ("bfloat16", "float32")))
register("Vogozen", ModelEntry(_vogozen_config, _hybrid_engine, ("bfloat16", "float32")))
