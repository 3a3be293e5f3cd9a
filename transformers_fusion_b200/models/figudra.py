"""Figudra: the stack model of parallel layers - softmax attention of two kinds or gated linear attention beside a dense or grouped
mixture-of-experts feed-forward - over a normed embedding, in which a layer may use the tensors of another.

The model folder holds ``config.json`` (``FigudraConfig.from_dict``) and ``model.safetensors``; a layer's tensors are l<i>.norm1,
l<i>.mix.* and l<i>.mlp.*, the experts l<i>.mlp.e<j>.* (``StackModel.named_tensors`` maps each to its place in the fused
parameters)."""
from __future__ import annotations

from ..ops import stack as K
from .config import FigudraConfig
from .stack import ParallelLayer, StackModel


class FigudraModel(StackModel):
    config_cls = FigudraConfig
    layer_cls = ParallelLayer
    kernel_units = K.UNITS_GATED
    embed_norm_name = "embed.norm"
