"""Lanedra: the stack model whose layers are differential sliding-window attention or the gated delta rule.

The model folder holds ``config.json`` (``LanedraConfig.from_dict``) and ``model.safetensors``; matrices are [out, in], a layer's
tensors are l<i>.norm*, l<i>.mix.* and l<i>.mlp.* (``StackModel.named_tensors`` maps each to its place in the fused
parameters)."""
from __future__ import annotations

from .config import LanedraConfig
from .stack import StackModel


class LanedraModel(StackModel):
    config_cls = LanedraConfig
