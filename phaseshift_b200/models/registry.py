"""Model families: what the engine and the applications need to know about a model, looked up by its ``config.json``.

A family names how to recognise its model directories, its random-init presets, how to build engine weights for either, and
the runner that executes one scheduled step.  Its configuration object carries the rest of the contract:
``vocab_size``, ``hidden_size``, ``eos_token_ids``, ``geometry(tp_rank, tp_size)``, ``state_specs(geometry)`` (cache and state
per layer execution, runtime/state.py) and ``family`` (the name it is registered under).
"""
from __future__ import annotations

import importlib
import json
from dataclasses import dataclass
from pathlib import Path
from typing import Callable, Dict, List

import torch


@dataclass(frozen=True)
class ModelFamily:
    name: str
    matches: Callable[[dict], bool]                  # parsed config.json -> is it ours
    config_from_dir: Callable
    presets: Callable[[], Dict[str, Callable]]       # random-init model name -> configuration factory
    load: Callable                                   # (model_dir, device, preset, dtype, **kw) -> engine weights
    random: Callable                                 # (cfg, device, preset, dtype, **kw) -> engine weights
    runner: Callable                                 # (weights, state, ops, tp) -> runner


DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class UnsupportedOption(ValueError):
    """A weight preset, precision or parallel layout that the model's family does not have."""


def _reject(cond: bool, what: str) -> None:
    if cond:
        raise UnsupportedOption(what)


# ---------------------------------------------------------------- Qwen3.5-style hybrid decoder
def _qwen_config(model_dir):
    from .qwen35.config import Qwen35Config
    return Qwen35Config.from_dir(model_dir)


def _qwen_presets():
    from .qwen35.config import PRESETS
    return PRESETS


def _qwen_dtype(device, dtype) -> None:
    _reject(dtype == torch.float32 and torch.device(device).type == "cuda", "the hybrid decoder has no 32-bit CUDA kernels")


def _qwen_load(model_dir, device, preset=None, dtype=None, **kw):
    from .qwen35.weights import load_engine_weights
    _qwen_dtype(device, dtype)
    return load_engine_weights(model_dir, device, preset, **kw)


def _qwen_random(cfg, device, preset=None, dtype=None, **kw):
    from .qwen35.weights import build_engine_weights, random_getter
    _qwen_dtype(device, dtype)
    return build_engine_weights(cfg, random_getter(cfg, 0, device), preset or "bf16", device, **kw)


def _qwen_runner(weights, state, ops, tp=None):
    from .qwen35.model import Qwen35Runner
    return Qwen35Runner(weights, state, ops, tp)


# ---------------------------------------------------------------- decoders with plain weights that run on one rank
def _plain_family(name: str, architecture: str) -> ModelFamily:
    """Family of ``models/<name>``: its modules ``config`` (<Architecture>Config, PRESETS), ``weights`` (load_engine_weights,
    build_engine_weights, random_getter) and ``model`` (<Architecture>Runner); bf16 or 32-bit weights, no tensor parallelism."""
    def module(which):
        return importlib.import_module(f".{name}.{which}", __package__)

    def options(preset, kw) -> None:
        _reject(preset not in (None, "bf16"), f"{architecture} models have no {preset!r} weight preset (bf16, or 32-bit with dtype=float32)")
        _reject(kw.get("tp_size", 1) != 1, f"{architecture} models run on one rank")

    def load(model_dir, device, preset=None, dtype=None, **kw):
        options(preset, kw)
        return module("weights").load_engine_weights(model_dir, device, dtype)

    def rand(cfg, device, preset=None, dtype=None, **kw):
        options(preset, kw)
        return module("weights").build_engine_weights(cfg, module("weights").random_getter(cfg, 0, device), device, dtype)

    return ModelFamily(name, lambda raw: raw.get("architecture") == architecture,
                       lambda d: getattr(module("config"), architecture + "Config").from_dir(d), lambda: module("config").PRESETS, load, rand,
                       lambda weights, state, ops, tp=None: getattr(module("model"), architecture + "Runner")(weights, state, ops, tp))


FAMILIES: List[ModelFamily] = [
    _plain_family("rotutar", "Rotutar"),
    _plain_family("fudulix", "Fudulix"),
    _plain_family("luvutar", "Luvutar"),
    _plain_family("gebuzen", "Gebuzen"),
    # the first family of the framework; a config.json without an architecture of another family is read as its own
    ModelFamily("qwen35", lambda raw: "architecture" not in raw, _qwen_config, _qwen_presets, _qwen_load, _qwen_random, _qwen_runner),
]


def family_by_name(name: str) -> ModelFamily:
    for f in FAMILIES:
        if f.name == name:
            return f
    raise ValueError(f"unknown model family {name!r}")


def family_of(cfg) -> ModelFamily:
    return family_by_name(cfg.family)


def family_of_dir(model_dir) -> ModelFamily:
    raw = json.loads((Path(model_dir) / "config.json").read_text())
    for f in FAMILIES:
        if f.matches(raw):
            return f
    raise ValueError(f"unknown architecture {raw.get('architecture')!r} in {model_dir}")


def preset_names() -> List[str]:
    return [n for f in reversed(FAMILIES) for n in f.presets()]


def preset_config(name: str):
    for f in FAMILIES:
        if name in f.presets():
            return f.presets()[name]()
    raise ValueError(f"unknown random-init model {name!r}")


def config_from_dir(model_dir):
    return family_of_dir(model_dir).config_from_dir(model_dir)


def load_weights(model_dir, device="cpu", preset=None, dtype=None, **kw):
    """Engine weights of a model directory of any family.  ``dtype``: torch.bfloat16 / torch.float32, None = the family's default."""
    return family_of_dir(model_dir).load(model_dir, device, preset, dtype, **kw)


def random_weights(cfg, device="cpu", preset=None, dtype=None, **kw):
    return family_of(cfg).random(cfg, device, preset, dtype, **kw)
