from .engine_config import EngineConfig
from .model_config import ConfigError, LuvutarConfig, MemilornConfig, PutelixConfig, Qwen2Config, SinoraxConfig, architecture_name, read_config_json

__all__ = ["ConfigError", "EngineConfig", "LuvutarConfig", "MemilornConfig", "PutelixConfig", "Qwen2Config", "SinoraxConfig", "architecture_name", "read_config_json"]
