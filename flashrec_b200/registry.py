"""Model registry: which model class a checkpoint directory's ``config.json`` names, and how it is loaded.

``lookup(config)`` -> :class:`ModelFamily`; ``load_model(path, dtype, device)`` -> a model with its weights. Families:
the FP8 Qwen3 of :mod:`flashrec_b200.decoder` and the 16/32-bit decoder models."""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Callable, List, Optional, Sequence

import torch


@dataclass(frozen=True)
class ModelFamily:
    name: str
    matches: Callable[[dict], bool]
    load: Callable[[str, dict, torch.dtype, object], object]  # (directory, config, dtype, device) -> model
    dtypes: Sequence[torch.dtype]
    sources: Optional[Sequence[str]] = None  # csrc stems a build for this family alone needs (None: all)


def _is_qwen3(cfg: dict) -> bool:
    return cfg.get("model_type") == "qwen3" or "Qwen3ForCausalLM" in (cfg.get("architectures") or [])


def _load_qwen3(path: str, cfg: dict, dtype: torch.dtype, device):
    from flashrec_b200.qwen3_lm import load_qwen3_lm

    return load_qwen3_lm(path, device)


def _load_dibepel(path: str, cfg: dict, dtype: torch.dtype, device):
    from flashrec_b200.dibepel import DibepelConfig, DibepelForCausalLM
    from flashrec_b200.weights import read_tensors

    return DibepelForCausalLM(DibepelConfig.from_json(cfg), read_tensors(path), dtype, device)


def _load_kotipel(path: str, cfg: dict, dtype: torch.dtype, device):
    from flashrec_b200.kotipel import KotipelConfig, KotipelForCausalLM
    from flashrec_b200.weights import read_tensors

    return KotipelForCausalLM(KotipelConfig.from_json(cfg), read_tensors(path), dtype, device)


FAMILIES: List[ModelFamily] = [
    ModelFamily("qwen3-fp8", _is_qwen3, _load_qwen3, (torch.bfloat16,)),
    ModelFamily("dibepel", lambda c: c.get("architecture") == "Dibepel", _load_dibepel, (torch.bfloat16, torch.float32),
                ("capi", "dense_proj", "lm_rows", "attn_mix", "attn_talk")),
    ModelFamily("kotipel", lambda c: c.get("architecture") == "Kotipel", _load_kotipel, (torch.bfloat16, torch.float32),
                ("capi", "dense_proj", "lm_rows", "attn_mix", "attn_talk", "linear_scan", "linear_chunk")),
]


def read_config(path: str) -> dict:
    return json.loads((Path(path) / "config.json").read_text(encoding="utf-8"))


def lookup(cfg: dict) -> ModelFamily:
    for f in FAMILIES:
        if f.matches(cfg):
            return f
    raise ValueError(f"no model family for architecture {cfg.get('architecture') or cfg.get('architectures')!r}")


def load_model(path: str, dtype: torch.dtype = torch.bfloat16, device="cuda:0"):
    cfg = read_config(path)
    family = lookup(cfg)
    if dtype not in family.dtypes:
        raise NotImplementedError(f"{family.name} does not run in {dtype}")
    return family.load(str(path), cfg, dtype, device)
