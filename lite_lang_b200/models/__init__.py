"""Architectures.  Importing this package registers each of them."""
from . import lenuzen, muduvik, nevurax, qwen2, redirax, rufisun, tusipel  # noqa: F401
from .lenuzen import LenuzenConfig
from .muduvik import MuduvikConfig
from .nevurax import NevuraxConfig
from .qwen2 import Qwen2Config
from .redirax import RediraxConfig
from .rufisun import RufisunConfig
from .tusipel import TusipelConfig

__all__ = ["LenuzenConfig", "MuduvikConfig", "NevuraxConfig", "Qwen2Config", "RediraxConfig", "RufisunConfig",
           "TusipelConfig"]
