"""Decoder families and how a checkpoint directory chooses one.

``detect(config)`` reads ``architecture`` / ``architectures`` / ``model_type`` of a parsed config.json; a :class:`Family` knows how
to load its weights and how to open a decoding session (``hidden`` over whole prompts, ``head``, ``step``, ``retain``)."""
from __future__ import annotations

import importlib
import json
import os
from dataclasses import dataclass
from typing import Callable, List, Optional, Tuple

import torch


@dataclass(frozen=True)
class Family:
    name: str
    architectures: Tuple[str, ...]             # prefixes, lower case
    module: str
    session_class: Optional[str] = None        # decoding session, for the families that share the protocol
    kernel_units: Optional[Tuple[str, ...]] = None      # csrc units of its inference path (None: not listed, use the whole library)
    loader: str = "load_pretrained"
    ragged: bool = False                       # one prefill takes prompts of different lengths

    def load(self, model_dir: str, device, dtype, log=None):
        m = importlib.import_module(f"tyr_b200.models.{self.module}")
        return getattr(m, self.loader)(model_dir, device, dtype, log)

    def session(self, model, batch: int, max_len: int):
        if self.session_class is None:
            raise ValueError(f"{self.name} has no decoding session")
        m = importlib.import_module(f"tyr_b200.models.{self.module}")
        return getattr(m, self.session_class)(model, batch, max_len)


FAMILIES: List[Family] = [
    Family("vonulix", ("vonulix",), "vonulix", "CacheSession",
           ("attention_fwd", "attention_general", "decode_attention", "decode_gemm", "depth_average", "embed", "gates", "gemm_tcgen05", "moe_nvfp4", "moe_stream",
            "norm", "rotary_store", "skinny_gemm"), ragged=True),
    Family("nizedra", ("nizedra",), "nizedra", "CacheSession",
           ("attention_fwd", "attention_general", "decode_gemm", "delta_general", "gemm_tcgen05", "joint_attention", "joint_tcgen05", "latent", "lightning", "mix_conv",
            "norm", "skinny_gemm"), ragged=True),
    Family("kinetar", ("kinetar",), "kinetar", "CacheSession",
           ("attention_fwd", "attention_general", "decode_attention", "decode_gemm", "delta_general", "delta_rule", "embed", "gemm_tcgen05", "mix_conv",
            "norm", "selective_scan", "skinny_gemm"), ragged=True),
    Family("zatorax", ("zatorax",), "zatorax", "CacheSession",
           ("attention_fwd", "attention_general", "decode_attention", "decode_gemm", "delta_general", "delta_rule", "gemm_tcgen05", "moe_nvfp4",
            "norm", "skinny_gemm"), ragged=True),
    Family("qwen35", ("qwen3_5", "qwen3.5", "qwen3_6", "qwen3.6"), "qwen35", "HybridCache"),
    Family("laguna", ("laguna",), "laguna", "CacheSession"),
    Family("gemma4", ("gemma4",), "gemma4"),
    Family("qwen25omni", ("qwen2_5_omni", "qwen2.5omni"), "qwen"),
    Family("qwen3", ("qwen3",), "qwen"),
]


def by_name(name: str) -> Family:
    for f in FAMILIES:
        if f.name == name:
            return f
    raise ValueError(f"unknown model family {name}; known: {', '.join(f.name for f in FAMILIES)}")


def detect(config: dict) -> Family:
    """The family of a parsed config.json (the first whose prefix matches: more specific families come first)."""
    names = [config.get("architecture"), config.get("model_type"), *(config.get("architectures") or [])]
    names = [str(n).lower() for n in names if n]
    for f in FAMILIES:
        if any(n.startswith(p) for n in names for p in f.architectures):
            return f
    raise ValueError(f"no model family for config.json with architecture {names or 'unnamed'}; known: {', '.join(f.name for f in FAMILIES)}")


def detect_dir(model_dir: str) -> Family:
    with open(os.path.join(model_dir, "config.json")) as f:
        return detect(json.load(f))
