"""B200-native block-diffusion decode path of MinerU-Diffusion's nano_dvlm engine.

The directory name carries a hyphen, so import it with
``importlib.import_module("mineru-diffusion_b200")``; after the first import the
alias ``mineru_diffusion_b200`` is registered too.
"""
import sys as _sys

from . import _lib, ops
from .decoder import DecoderEngine, DecoderWeights, LayerWeights
from .hybrid import HybridEngine, HybridWeights
from .loader import load_decoder_weights, load_hybrid_weights
from .engine import (BlockManager, CausalScheduler, CausalSequence, Config, Context, DecoderConfig, HybridConfig,
                     SamplingParams, Scheduler, Sequence, SequenceStatus, StateManager)
from .engine.llm_engine import LLMEngine
from .engine.model_runner import ModelRunner
from .engine.causal_runner import CausalModelRunner

_sys.modules.setdefault("mineru_diffusion_b200", _sys.modules[__name__])

__all__ = ["ops", "DecoderEngine", "DecoderWeights", "LayerWeights", "HybridEngine", "HybridWeights", "load_decoder_weights",
           "load_hybrid_weights", "BlockManager", "Config", "Context", "DecoderConfig", "HybridConfig", "SamplingParams",
           "Scheduler", "CausalScheduler", "Sequence", "CausalSequence", "SequenceStatus", "StateManager", "LLMEngine",
           "ModelRunner", "CausalModelRunner"]
