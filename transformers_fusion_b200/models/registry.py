"""Model classes by architecture name, and model folders (config.json + safetensors).

``load_folder`` builds the class that a folder's config.json names and fills it through the native safetensors reader;
``load_any`` also takes a ``.quant`` container.  The command-line tools and the trace runner open models through these."""
from __future__ import annotations

import importlib
import inspect
import json
import os
from typing import Dict, Tuple

import torch

# architecture -> (module, model class); the class names its configuration in ``config_cls``
ARCHITECTURES: Dict[str, Tuple[str, str]] = {
    "Lanedra": ("lanedra", "LanedraModel"),
    "Tekenex": ("tekenex", "TekenexModel"),
    "Figudra": ("figudra", "FigudraModel"),
    "Toderax": ("toderax", "ToderaxModel"),
}


def register(architecture: str, module: str, cls: str):
    """Add a model class (``module`` relative to this package, or an absolute module name)."""
    ARCHITECTURES[architecture] = (module, cls)


def model_class(architecture: str):
    if architecture not in ARCHITECTURES:
        raise ValueError(f"unknown architecture '{architecture}' (known: {', '.join(sorted(ARCHITECTURES))})")
    module, cls = ARCHITECTURES[architecture]
    return getattr(importlib.import_module("." + module if "." not in module else module, __package__), cls)


def is_folder(path) -> bool:
    return os.path.isdir(path) and os.path.exists(os.path.join(path, "config.json"))


def read_config(path):
    """(model class, configuration) of a model folder."""
    with open(os.path.join(path, "config.json")) as f:
        d = json.load(f)
    if "architecture" not in d:
        raise ValueError(f"{path}: config.json names no architecture")
    cls = model_class(d["architecture"])
    if "shapes" not in inspect.signature(cls.config_cls.from_dict).parameters:
        return cls, cls.config_cls.from_dict(d)
    from ..quant.importers import _sources
    shapes = {}                      # sizes that only the tensors give
    for src in _sources(path):
        shapes.update((n, tuple(src.shape(n))) for n in src.names)
        src.close()
    return cls, cls.config_cls.from_dict(d, shapes=shapes)


def load_folder(path, device="cpu", dtype=torch.float32):
    """The model of a folder with its weights.  Every tensor of the model has to be in the folder with the shape the
    configuration gives, and the folder may hold no others."""
    from ..quant.importers import _sources
    cls, cfg = read_config(path)
    model = cls(cfg, device=device, dtype=dtype, seed=None)
    left = dict(model.named_tensors())
    with torch.no_grad():
        for src in _sources(path):
            for name in src.names:
                if name not in left:
                    raise ValueError(f"{path}: unexpected tensor {name}")
                dst = left.pop(name)
                if tuple(src.shape(name)) != tuple(dst.shape):
                    raise ValueError(f"{name}: {tuple(src.shape(name))} in the file, {tuple(dst.shape)} expected")
                dst.copy_(src.read(name).to(dst.dtype))
            src.close()
    if left:
        raise KeyError(f"{path}: tensor {sorted(left)[0]} missing")
    model.finalize()
    return model


def limit_build(path):
    """For a process that only runs the forward passes of this folder's model: a kernel library that still has to be built is
    built from the translation units of that model's passes alone."""
    from ..ops import _lib
    with open(os.path.join(path, "config.json")) as f:
        cls = model_class(json.load(f)["architecture"])
    _lib.need_units(f"tfb_kernels_{cls.__name__.lower()}", cls.kernel_units)


def load_any(path, device="cpu", dtype=torch.float32):
    """A model folder or a ``.quant`` container."""
    if is_folder(path):
        return load_folder(path, device, dtype)
    from ..quant import codec
    return codec.load_model(path, device=device, dtype=dtype)


def save_folder(model, path):
    """config.json and model.safetensors (bf16) of a stack model."""
    import struct
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(model.cfg.to_dict(), f, indent=1)
    head, off, blobs = {}, 0, []
    for name, t in model.named_tensors():
        raw = t.detach().to("cpu", torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        off += len(raw)
        blobs.append(raw)
    h = json.dumps(head).encode()
    h += b" " * (-len(h) % 8)
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h)
        for raw in blobs:
            f.write(raw)
