from .model_config import ModelConfig, ConfigError, DEFAULT_ARCHITECTURE
from .munevik_config import MunevikConfig
from .mizupel_config import MizupelConfig
from .mokalorn_config import MokalornConfig
from .dabilorn_config import DabilornConfig
from .renanex_config import RenanexConfig
from .fokurax_config import FokuraxConfig
from .engine_config import CacheConfig, SchedulerConfig, EngineConfig, COMPUTE_DTYPES

__all__ = ["ModelConfig", "MunevikConfig", "MizupelConfig", "MokalornConfig", "DabilornConfig", "RenanexConfig", "FokuraxConfig", "ConfigError", "DEFAULT_ARCHITECTURE", "CacheConfig", "SchedulerConfig",
           "EngineConfig", "COMPUTE_DTYPES"]
