from .errors import ConfigError, MissingKey, InvalidValue, UnknownArchitecture
from .registry import (register_architecture, architecture_for, known_architectures,
                       load_config, read_config_json, architecture_name)
from .qwen2 import Qwen2Config
from .rifizen import RifizenConfig
from .vilulorn import VilulornConfig
from .figalix import FigalixConfig
from .ludusun import LudusunConfig
from .gedilorn import GedilornConfig
from .dubodra import DubodraConfig
from . import vilulorn   # (its builder registers "Vilulorn")
