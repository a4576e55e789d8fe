"""Model registry: what a config.json (or a preset name) is, and how its weights and its serving forward pass are made.

A family is found by the "architecture" / "architectures" key of config.json; without one the folder is a Hugging Face
Llama checkpoint."""
from __future__ import annotations

import copy
import json
from dataclasses import dataclass
from pathlib import Path
from typing import Callable

import torch

from . import config as llama_config
from . import latanex, logozen, ridazen, sigosun


@dataclass(frozen=True)
class Family:
    name: str
    config_cls: type
    presets: dict
    load_config: Callable                  # directory -> config
    load_weights: Callable                 # (cfg, directory, device, dtype) -> weights of one rank
    random_weights: Callable               # (cfg, device, dtype, seed) -> weights of one rank
    runner: Callable                       # () -> serving runner class
    dtypes: tuple                          # compute dtypes that have CUDA kernels


def _llama_weights(cfg, directory, device, dtype):
    from ..serve.model_runner import TPWeights
    from .hf_io import load_resident
    _, full = load_resident(directory, "cpu", dtype)
    return TPWeights(cfg, 0, 1, device, dtype).load_from_full(full)


def _llama_random(cfg, device, dtype, seed=0):
    from ..serve.model_runner import TPWeights
    return TPWeights(cfg, 0, 1, device, dtype).init_random(seed)


def _llama_runner():
    from ..serve.model_runner import ModelRunner
    return ModelRunner


def _stack_runner():
    from ..serve.stack_runner import StackRunner
    return StackRunner


FAMILIES: dict[str, Family] = {
    "LlamaForCausalLM": Family("LlamaForCausalLM", llama_config.LlamaConfig, llama_config.PRESETS, llama_config.LlamaConfig.load,
                               _llama_weights, _llama_random, _llama_runner, (torch.bfloat16, torch.float16)),
    sigosun.ARCHITECTURE: Family(
        sigosun.ARCHITECTURE, sigosun.SigosunConfig, sigosun.PRESETS, sigosun.SigosunConfig.load, sigosun.load_weights,
        lambda cfg, device, dtype, seed=0: sigosun.from_state(cfg, sigosun.random_state(cfg, seed, device), device, dtype),
        _stack_runner, (torch.bfloat16, torch.float32)),
    logozen.ARCHITECTURE: Family(
        logozen.ARCHITECTURE, logozen.LogozenConfig, logozen.PRESETS, logozen.LogozenConfig.load, logozen.load_weights,
        lambda cfg, device, dtype, seed=0: logozen.from_state(cfg, logozen.random_state(cfg, seed, device), device, dtype),
        _stack_runner, (torch.bfloat16, torch.float32)),
    latanex.ARCHITECTURE: Family(
        latanex.ARCHITECTURE, latanex.LatanexConfig, latanex.PRESETS, latanex.LatanexConfig.load, latanex.load_weights,
        lambda cfg, device, dtype, seed=0: latanex.from_state(cfg, latanex.random_state(cfg, seed, device), device, dtype),
        _stack_runner, (torch.bfloat16, torch.float32)),
    ridazen.ARCHITECTURE: Family(
        ridazen.ARCHITECTURE, ridazen.RidazenConfig, ridazen.PRESETS, ridazen.RidazenConfig.load, ridazen.load_weights,
        lambda cfg, device, dtype, seed=0: ridazen.from_state(cfg, ridazen.random_state(cfg, seed, device), device, dtype),
        _stack_runner, (torch.bfloat16, torch.float32)),
}


def family_of(cfg) -> Family:
    for f in FAMILIES.values():
        if isinstance(cfg, f.config_cls):
            return f
    raise ValueError(f"no model family for configuration {type(cfg).__name__}")


def config_from_dir(directory: str | Path):
    with open(Path(directory) / "config.json") as f:
        d = json.load(f)
    names = [d["architecture"]] if "architecture" in d else d.get("architectures") or ["LlamaForCausalLM"]
    for n in names:
        if n in FAMILIES:
            return FAMILIES[n].load_config(directory)
    raise ValueError(f"unsupported architecture {names} (known: {sorted(FAMILIES)})")


def preset(name: str):
    for f in FAMILIES.values():
        if name in f.presets:
            return copy.deepcopy(f.presets[name])
    return None
