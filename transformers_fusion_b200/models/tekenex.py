"""Tekenex: the stack model of latent attention layers with dense or mixture-of-experts feed-forwards, normed on the output of
every sublayer only, whose head is the embedding table.

The model folder holds ``config.json`` (``TekenexConfig.from_dict``) and ``model.safetensors``; a layer's tensors are l<i>.norm1,
l<i>.ls1, l<i>.mix.* and so on, the experts l<i>.mlp.e<j>.* (``StackModel.named_tensors`` maps each to its place in the fused
parameters)."""
from __future__ import annotations

from ..ops import stack as K
from .config import TekenexConfig
from .stack import OutputNormLayer, StackModel


class TekenexModel(StackModel):
    config_cls = TekenexConfig
    layer_cls = OutputNormLayer
    kernel_units = K.UNITS_LATENT
