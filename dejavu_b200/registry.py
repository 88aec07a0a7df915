"""Model registry: which class serves a model folder (config.json + .safetensors), chosen by the configuration.

    model = load_model("path/to/model", dtype=torch.bfloat16, device="cuda")

An architecture is the value of config.json's "architecture", or the first of its "architectures" (Hugging Face
folders). Each entry names the dtypes it runs in, the shared library its kernels are in, and a function that builds and
fills the model.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable

import torch


@dataclass(frozen=True)
class Entry:
    build: Callable  # (config dict, tensors, device, dtype) -> model, weights loaded
    dtypes: tuple
    library: str     # name in dejavu_b200.build.LIBS


def _build_ninolorn(raw, tensors, device, dtype):
    from .ninolorn import NinolornForCausalLM

    shapes = {k: tuple(v.shape) for k, v in tensors.items()}
    return NinolornForCausalLM(raw, shapes, device=device, dtype=dtype).load_tensors(tensors)


def _build_tifosun(raw, tensors, device, dtype):
    from .tifosun import TifosunForCausalLM

    return TifosunForCausalLM(raw, device=device, dtype=dtype).load_tensors(tensors)


def opt_config_from_json(raw):
    """Hugging Face OPT config.json -> this package's OPT configuration (dense: every head and neuron)."""
    from .gpt import opt_config

    if not raw.get("do_layer_norm_before", True) or raw.get("word_embed_proj_dim", raw["hidden_size"]) != raw["hidden_size"]:
        raise ValueError("only pre-norm OPT decoders without an embedding projection are supported")
    d = raw["hidden_size"]
    return opt_config("opt-125m", model_name=raw.get("_name_or_path", "opt"), n_layer=raw["num_hidden_layers"], n_embd=d,
                      hidden_size=d, n_head=raw["num_attention_heads"], n_inner=raw["ffn_dim"],
                      vocab_size=raw["vocab_size"], n_positions=raw["max_position_embeddings"],
                      max_position_embeddings=raw["max_position_embeddings"], mlp_K=raw["ffn_dim"],
                      att_K=[raw["num_attention_heads"]] * 2, activation_function=raw.get("activation_function", "relu"))


def _build_opt(raw, tensors, device, dtype):
    from .checkpoint import remap_state_dict_opt, shard_state_dict_tp
    from .gpt import GPTLMHeadModel

    cfg = opt_config_from_json(raw)
    tensors = {(k if k.startswith(("model.", "lm_head")) else "model." + k): v.to(dtype) for k, v in tensors.items()}
    model = GPTLMHeadModel(cfg, device=device, dtype=dtype)
    model.load_state_dict(shard_state_dict_tp(remap_state_dict_opt(tensors, cfg), cfg, 1, 0))
    return model


MODELS = {
    "Ninolorn": Entry(_build_ninolorn, (torch.bfloat16, torch.float32), "hybrid"),
    "Tifosun": Entry(_build_tifosun, (torch.bfloat16, torch.float32), "routed"),
    "OPTForCausalLM": Entry(_build_opt, (torch.float16,), "sparse"),
}


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def entry_for(raw: dict) -> Entry:
    name = raw.get("architecture") or (raw.get("architectures") or [None])[0]
    if name not in MODELS:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(MODELS)}")
    return MODELS[name]


def load_model(folder: str, dtype=None, device="cuda"):
    """The model of a folder, weights loaded, ready to generate. dtype None: the first its class runs in."""
    from .checkpoint import read_model_tensors

    raw = read_config(folder)
    entry = entry_for(raw)
    dtype = dtype or entry.dtypes[0]
    if dtype not in entry.dtypes:
        raise ValueError(f"this model runs in {[str(d) for d in entry.dtypes]}, not {dtype}")
    return entry.build(raw, read_model_tensors(folder), torch.device(device), dtype).eval()
