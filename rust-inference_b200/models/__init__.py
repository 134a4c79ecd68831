"""Architectures.  Importing this package registers them."""
from . import gotulorn, kagatar, pitenex, puratar, qwen3, ranudra, zavevik  # noqa: F401
from .gotulorn import GotulornConfig
from .kagatar import KagatarConfig
from .pitenex import PitenexConfig
from .puratar import PuratarConfig
from .qwen3 import Qwen3Config
from .ranudra import RanudraConfig
from .zavevik import ZavevikConfig

__all__ = ["GotulornConfig", "KagatarConfig", "PitenexConfig", "PuratarConfig", "Qwen3Config", "RanudraConfig", "ZavevikConfig"]
