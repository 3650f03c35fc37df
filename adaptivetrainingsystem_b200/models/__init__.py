from .transformer import (DeepSeekTransformer, TransformerBlock, GroupedQueryAttention, DenseSwiGLU, SwiGLUExpert,
                          MoEFFNLayer, MoDRouter, MoDFFN, RMSNorm, LayerNorm, RotaryEmbedding, KVCache,
                          estimate_parameters)
from ..config import ModelConfig, DeepSeekConfig
from ..config import LayerSpec, NemipelConfig, VimodraConfig
from .cache import LayerStateCache, SequenceCache
from .layered import LayeredDecoder
from .nemipel import Nemipel
from .vimodra import Vimodra
from .registry import MODELS, ModelEntry, load_model, read_config, register_model
