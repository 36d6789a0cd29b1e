"""The model families of the framework: ``config.json``'s ``architecture`` -> configuration, weights, runner.

A model folder holds ``config.json`` and ``model.safetensors``.  ``load_model`` picks the family by the
architecture's name; the serving engine asks the family for its runner (the layer pipeline and the cache of
that family) and does everything else itself.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, fields
from pathlib import Path
from typing import Any, Callable

import torch

from ..ckpt.safetensors import load_safetensors
from ..config import ModelConfig
from .lisunex import LisunexConfig, LisunexModel
from .llama import KotodamaModel
from .vunitar import VunitarConfig, VunitarModel


@dataclass(frozen=True)
class Family:
    config: Callable[[dict], Any]                                  # config.json -> configuration
    model: Callable[[Any, dict[str, torch.Tensor]], Any]           # configuration, weights -> model
    random: Callable[[Any, int], Any]                              # configuration, seed -> randomly initialised model
    model_type: type                                               # what the serving engine is handed
    runner: str                                                    # class in kotodama_b200.serve.runners
    native_sources: tuple[str, ...]                                # csrc files that serving this family needs


def _llama_config(d: dict) -> ModelConfig:
    known = {f.name for f in fields(ModelConfig)}
    return ModelConfig(**{k: v for k, v in d.items() if k in known})


def _llama_model(cfg: ModelConfig, weights: dict[str, torch.Tensor]) -> KotodamaModel:
    from ..ckpt.manager import clean_state_dict
    m = KotodamaModel(cfg)
    m.load_state_dict(clean_state_dict(weights), strict=True)
    return m


def _llama_random(cfg: ModelConfig, seed: int) -> KotodamaModel:
    torch.manual_seed(seed)
    return KotodamaModel(cfg)


FAMILIES: dict[str, Family] = {
    "Kotodama": Family(_llama_config, _llama_model, _llama_random, KotodamaModel, "LlamaRunner", ()),
    "Vunitar": Family(VunitarConfig.from_dict, VunitarModel, VunitarModel.random_init, VunitarModel, "LatentRunner",
                      ("elementwise", "serve", "sampler", "attn_sm100", "gemm_sm100", "gemm2_sm100", "gemm_skinny_sm100",
                       "latent_attn", "latent_attn_sm100", "moe", "gemm_grouped_sm100", "gemm_f32", "block")),
    "Lisunex": Family(LisunexConfig.from_dict, LisunexModel, LisunexModel.random_init, LisunexModel, "HybridRunner",
                      ("elementwise", "serve", "sampler", "attn_sm100", "gemm_sm100", "gemm2_sm100", "gemm_skinny_sm100",
                       "gemm_f32", "block", "paged_attn", "delta", "delta_sm100")),
}


def family_of(model: Any) -> Family:
    for f in FAMILIES.values():
        if isinstance(model, f.model_type):
            return f
    raise TypeError(f"no registered model family for {type(model).__name__}")


def read_config(folder: str | Path) -> tuple[Family, Any]:
    d = json.loads((Path(folder) / "config.json").read_text())
    name = d.get("architecture")
    if name not in FAMILIES:
        raise ValueError(f"unknown architecture {name!r}; registered: {sorted(FAMILIES)}")
    return FAMILIES[name], FAMILIES[name].config(d)


def load_model(folder: str | Path) -> Any:
    family, cfg = read_config(folder)
    return family.model(cfg, load_safetensors(Path(folder) / "model.safetensors"))
