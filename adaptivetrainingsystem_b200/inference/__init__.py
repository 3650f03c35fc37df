from .engine import GenerationEngine, SamplingParams, KVSlotManager, sample_next, GENERATION_MODES
from .pool import SequencePool
from .scheduler import ContinuousBatcher, Request
from .pipeline_generate import PipelineGenerator
from .trace import TraceRunner
