from .config import Config, DecoderConfig
from .hybrid_config import HybridConfig
from .sampling_params import SamplingParams
from .sequence import Sequence, SequenceStatus
from .block_manager import BlockManager
from .scheduler import Scheduler
from .context import Context
from .causal_scheduler import CausalScheduler, CausalSequence
from .state_manager import StateManager

__all__ = ["Config", "DecoderConfig", "SamplingParams", "Sequence", "SequenceStatus", "BlockManager",
           "Scheduler", "Context", "HybridConfig", "CausalScheduler", "CausalSequence", "StateManager"]
