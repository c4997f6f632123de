"""Model designs the engine serves.

A ``config.json`` names its design in ``architecture`` (the block-diffusion decoder's carries none).  An entry says how
that file is read and which model runner and scheduler drive the design; everything else of the engine is shared.
"""
from __future__ import annotations

from dataclasses import dataclass
from importlib import import_module
from typing import Callable

from .hybrid_config import DESIGNS, HybridConfig


@dataclass(frozen=True)
class Architecture:
    name: str
    config_type: type
    read_config: Callable[[dict], object]     # parsed config.json -> config_type
    runner: str                               # "module:class", imported on first use
    scheduler: str
    request: str                              # makes a request from (token ids, SamplingParams, Config)

    def load(self, which: str):
        module, name = getattr(self, which).split(":")
        return getattr(import_module(module, __package__), name)


_BY_NAME: dict[str, Architecture] = {}


def register(arch: Architecture) -> None:
    _BY_NAME[arch.name] = arch


def by_name(name: str) -> Architecture:
    if name not in _BY_NAME:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(_BY_NAME))}")
    return _BY_NAME[name]


def of_config(decoder_config) -> Architecture:
    """The design a decoder configuration belongs to (the block-diffusion decoder if nothing else)."""
    return by_name(getattr(decoder_config, "architecture", "sdar"))


def _read_sdar(raw: dict):
    from types import SimpleNamespace
    from .config import DecoderConfig
    text = raw.get("language_model_config") or raw.get("text_config") or raw
    return DecoderConfig.from_namespace(SimpleNamespace(**text))


def read_config(raw: dict):
    """Decoder configuration of a parsed ``config.json``."""
    name = raw.get("architecture")
    return by_name(name).read_config(raw) if name is not None else _read_sdar(raw)


def sdar_request(token_ids, params, config):
    from .sequence import Sequence
    return Sequence(token_ids, params, denoising_block_size=config.block_size, mask_token_id=config.mask_token_id)


def causal_request(token_ids, params, config):
    from .causal_scheduler import CausalSequence
    return CausalSequence(token_ids, params)


register(Architecture("sdar", object, _read_sdar, ".model_runner:ModelRunner", ".scheduler:Scheduler",
                      ".registry:sdar_request"))
for _name in DESIGNS:
    register(Architecture(_name, HybridConfig, HybridConfig.from_json, ".causal_runner:CausalModelRunner",
                          ".causal_scheduler:CausalScheduler", ".registry:causal_request"))
