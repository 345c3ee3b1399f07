from .model_config import ConfigError, GqaMtpConfig, KefisunConfig, MizidraConfig, BiruvikConfig, KubolornConfig, LomutarConfig, TazadraConfig, read_config_json, write_config_json, UPSTREAM_ALIASES
from .engine_config import EngineConfig

__all__ = ["ConfigError", "GqaMtpConfig", "KefisunConfig", "MizidraConfig", "BiruvikConfig", "KubolornConfig", "LomutarConfig", "TazadraConfig", "EngineConfig", "read_config_json", "write_config_json",
           "UPSTREAM_ALIASES"]
