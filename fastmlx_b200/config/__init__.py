from .base import ConfigError, ModelConfig, parse_config_json, read_config_json
from .bonerax import BoneraxConfig
from .gekavik import GekavikConfig
from .gepadra import GepadraConfig
from .kafepel import KafepelConfig
from .llama import LlamaConfig, RopeScaling, YarnScaling
from .medirax import MediraxConfig
from .sorupel import SorupelConfig

__all__ = ["ConfigError", "ModelConfig", "LlamaConfig", "MediraxConfig", "GekavikConfig", "SorupelConfig", "KafepelConfig", "BoneraxConfig", "GepadraConfig", "RopeScaling", "YarnScaling",
           "parse_config_json", "read_config_json"]
