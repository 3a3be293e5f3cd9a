"""Toderax: the stack model of hyper-connected layers - HGRN2, or chunked attention and retention side by side - with mixtures of clamped
experts.

The model folder holds ``config.json`` (``ToderaxConfig.from_dict``) and ``model.safetensors``; a layer's tensors are l<i>.norm<q>,
l<i>.hc<q>.*, l<i>.mix.* (of two mixers l<i>.mix.left.* and l<i>.mix.right.*) and l<i>.mlp.*, the experts l<i>.mlp.e<j>.*
(``StackModel.named_tensors`` maps each to its place in the fused parameters)."""
from __future__ import annotations

from ..ops import stack as K
from .config import ToderaxConfig
from .stack import StackModel, StreamLayer, StreamResidual


class ToderaxModel(StreamResidual, StackModel):
    config_cls = ToderaxConfig
    layer_cls = StreamLayer
    kernel_units = K.UNITS_STREAMS
