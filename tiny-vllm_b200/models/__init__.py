"""Architectures of the package; importing a module registers its architecture."""

from . import bimolix, fezavik, gumapel, kelasun, lasupel, qwen3, zifunex  # noqa: F401
from .bimolix import BimolixConfig
from .fezavik import FezavikConfig
from .gumapel import GumapelConfig
from .kelasun import KelasunConfig
from .lasupel import LasupelConfig
from .qwen3 import Qwen3Config
from .zifunex import ZifunexConfig

__all__ = ["BimolixConfig", "FezavikConfig", "GumapelConfig", "KelasunConfig", "LasupelConfig",
           "Qwen3Config", "ZifunexConfig"]
