"""The models this package serves, and how a model directory becomes a decoder.

An entry names the shared library a model needs, how its checkpoint is read,
the decoder class and the compute types it offers.  ``config.json`` chooses the
entry: ``architecture`` (or the first of ``architectures``).
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable

from .spec import DESIGN_MIXERS, HybridSpec
from .weights import load_hybrid_weights, load_qwen3_weights


@dataclass(frozen=True)
class ModelEntry:
    name: str
    library: str                     # of csrc/build.py
    dtypes: tuple
    load_weights: Callable           # (model_dir, max_seq_len=, device=) -> dict
    make_decoder: Callable           # (weights, max_seq_len, max_prefill_len, dtype, device) -> DecodeEngine


def _qwen3_decoder(w, max_seq_len, max_prefill_len, dtype, device):
    from .decoder import MegakernelDecoder
    return MegakernelDecoder(w["embed_weight"], w["layer_weights"], w["final_norm_weight"], w["lm_head_weight"], w["cos_table"],
                             w["sin_table"], len(w["layer_weights"]) // 11, max_seq_len, max_prefill_len)


def _hybrid_decoder(w, max_seq_len, max_prefill_len, dtype, device):
    from .hybrid import HybridDecoder
    return HybridDecoder(w, max_seq_len, max_prefill_len, dtype=dtype, device=device)


MODELS = {
    "Qwen3ForCausalLM": ModelEntry("Qwen3ForCausalLM", "qwen3", ("bfloat16",), load_qwen3_weights, _qwen3_decoder),
    **{name: ModelEntry(name, "hybrid", ("bfloat16", "float32"), load_hybrid_weights, _hybrid_decoder) for name in DESIGN_MIXERS},
}


def architecture_of(cfg: dict) -> str:
    if "architecture" in cfg:
        return cfg["architecture"]
    if cfg.get("architectures"):
        return cfg["architectures"][0]
    return "Qwen3ForCausalLM"        # checkpoints of the reference's loader name none


def find_model(model_dir: str) -> ModelEntry:
    """The entry of a local model directory; the built-in synthetic weights are Qwen3's."""
    path = os.path.join(model_dir, "config.json")
    if not os.path.exists(path):
        return MODELS["Qwen3ForCausalLM"]        # its loader knows the synthetic names and reports a missing directory
    with open(path) as fh:
        name = architecture_of(json.load(fh))
    if name not in MODELS:
        raise ValueError(f"{path}: unknown architecture {name!r}; known: {', '.join(sorted(MODELS))}")
    return MODELS[name]


def build_decoder(model_name: str = "Qwen/Qwen3-0.6B", max_seq_len: int = 2048, max_prefill_len: int | None = None, weights: dict | None = None,
                  dtype: str = "bfloat16", device="cuda"):
    """(decoder, tokenizer or None) of a model directory, or of a weight dict of either kind."""
    if weights is None:
        entry = find_model(model_name)
        weights = entry.load_weights(model_name, max_seq_len=max_seq_len, device=device)
    else:
        spec = weights.get("spec")
        entry = MODELS[spec.architecture if isinstance(spec, HybridSpec) else "Qwen3ForCausalLM"]
    if dtype not in entry.dtypes:
        raise ValueError(f"{entry.name} runs in {', '.join(entry.dtypes)}, not {dtype}")
    decoder = entry.make_decoder(weights, max_seq_len, max_seq_len if max_prefill_len is None else max_prefill_len, dtype, device)
    return decoder, weights.get("tokenizer")
