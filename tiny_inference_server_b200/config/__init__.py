from .model_config import ConfigError, GqaMtpConfig, KefisunConfig, MizidraConfig, BiruvikConfig, KubolornConfig, LomutarConfig, read_config_json, write_config_json, UPSTREAM_ALIASES
from .engine_config import EngineConfig

__all__ = ["ConfigError", "GqaMtpConfig", "KefisunConfig", "MizidraConfig", "BiruvikConfig", "KubolornConfig", "LomutarConfig", "EngineConfig", "read_config_json", "write_config_json",
           "UPSTREAM_ALIASES"]
