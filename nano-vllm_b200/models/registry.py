"""Which model class serves a configuration, and how a config.json becomes one."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, fields

from .mupulorn import MupulornConfig, MupulornForCausalLM
from .qwen3 import Qwen3ForCausalLM
from .vekerax import VekeraxConfig, VekeraxForCausalLM


@dataclass
class ModelConfig:
    """The fields of a HF Qwen3 config the model reads (nanovllm/models/qwen3.py:127-143,167-171,199-203)."""
    hidden_size: int
    num_attention_heads: int
    num_key_value_heads: int
    head_dim: int
    intermediate_size: int
    num_hidden_layers: int
    vocab_size: int
    rms_norm_eps: float = 1e-6
    rope_theta: float = 1e6
    max_position_embeddings: int = 40960
    tie_word_embeddings: bool = False
    attention_bias: bool = False
    hidden_act: str = "silu"
    rope_scaling: dict | None = None
    eos_token_id: int | None = None

    architecture = "Qwen3ForCausalLM"

    @classmethod
    def from_dict(cls, d: dict) -> "ModelConfig":
        known = {f.name for f in fields(cls)}
        kept = {k: v for k, v in d.items() if k in known}
        kept.setdefault("head_dim", d["hidden_size"] // d["num_attention_heads"])
        if isinstance(kept.get("eos_token_id"), list):
            kept["eos_token_id"] = kept["eos_token_id"][0]
        return cls(**kept)

    @property
    def logits_size(self) -> int:
        return self.vocab_size


# architecture name -> (configuration class, model class)
REGISTRY = {
    "Qwen3ForCausalLM": (ModelConfig, Qwen3ForCausalLM),
    "Vekerax": (VekeraxConfig, VekeraxForCausalLM),
    "Mupulorn": (MupulornConfig, MupulornForCausalLM),
}


def config_from_dict(d: dict):
    name = d.get("architecture") or (d.get("architectures") or [None])[0]
    if name not in REGISTRY:
        raise ValueError(f"no model for architecture {name!r}; known: {sorted(REGISTRY)}")
    return REGISTRY[name][0].from_dict(d)


def load_config(model_dir: str):
    with open(os.path.join(model_dir, "config.json")) as f:
        return config_from_dict(json.load(f))


def build_model(config):
    return REGISTRY[config.architecture][1](config)
