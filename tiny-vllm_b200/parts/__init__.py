"""The parts a model is put together from, and their registries."""

from . import (attention, block, delta_rule, embedding, hyper, mlp, norm, parallel,  # noqa: F401  (they
               recurrent_unit, retention, rope, selective_scan)                     # register themselves)
from .base import Block, BuildContext, KVNeed, ParamSource, ParamSpec, Part, StateNeed
from .registry import build_part, part_kinds, register_part

__all__ = ["Block", "BuildContext", "KVNeed", "ParamSource", "ParamSpec", "Part", "StateNeed",
           "build_part", "part_kinds", "register_part"]
