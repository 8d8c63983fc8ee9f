"""Architectures this framework serves. Importing the package registers them."""

from . import diderax, fegilix, gasavik, guzovik, qwen3, risonex, sanevik  # noqa: F401  (each registers its architecture)
from .diderax import DideraxConfig
from .fegilix import FegilixConfig
from .gasavik import GasavikConfig
from .guzovik import GuzovikConfig
from .qwen3 import Qwen3Config
from .risonex import RisonexConfig
from .sanevik import SanevikConfig

__all__ = ["DideraxConfig", "FegilixConfig", "GasavikConfig", "GuzovikConfig", "Qwen3Config", "RisonexConfig", "SanevikConfig"]
