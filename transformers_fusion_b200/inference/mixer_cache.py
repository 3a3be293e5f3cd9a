"""What a decoder of mixed layers remembers of its sequences.

* Attention layers that have keys and values of their own: paged pools, one row of keys ([kv_heads, maps * dim]) and one of
  values per token, with the page allocator and block tables of ``kv_cache``; the layers share one page list per
  sequence.  When every attention layer looks back over a window, or to the start of its chunk of positions, pages that no layer will
  look at again go back to the allocator (``first_live_page``), and a prompt's earlier tokens are never written; the pages of the first
  tokens stay when some layer keeps them in sight (``kept_pages``).
* Latent attention layers: one paged pool with a row of ``latent_width`` entries per token (the latent, zeros behind it), under the
  same page list.
* Recurrent layers: a slot per sequence with the fp32 state matrices and, where there is one, the last inputs of the short convolution.  A slot's
  contents are only read by a sequence that goes on; a sequence that starts ignores and overwrites them, so slots need no
  clearing when they change hands.

A layer of two mixers side by side has what each of them needs, under the layer's index.

Because a recurrent state belongs to one point of one sequence, pages cannot be shared between sequences by prompt prefix
(``shareable`` is False for models with such layers, and for windowed caches, whose early pages are gone)."""
from __future__ import annotations

from typing import Dict, List

import torch

from ..models.config import first_key, mixers_of
from .kv_cache import PAGE, PageAllocator


class MixerCache:
    def __init__(self, cfg, num_pages: int, num_slots: int, dtype=torch.bfloat16, device="cuda"):
        self.cfg, self.num_pages, self.num_slots, self.dtype, self.device = cfg, num_pages, num_slots, dtype, torch.device(device)
        self.allocator = PageAllocator(num_pages)
        self.free_slots: List[int] = list(range(num_slots - 1, -1, -1))
        self.window = cfg.window
        self.kept_pages = (getattr(cfg, "keep_first", 0) + PAGE - 1) // PAGE if self.window else 0
        self.k: Dict[int, torch.Tensor] = {}
        self.v: Dict[int, torch.Tensor] = {}
        self.latent: Dict[int, torch.Tensor] = {}
        self.state: Dict[int, torch.Tensor] = {}
        self.conv: Dict[int, torch.Tensor] = {}
        parts = [(i, m) for i, l in enumerate(cfg.layers) for m in mixers_of(l.mixer)]
        self.looks_back = sorted({(m.window, getattr(m, "chunk", 0)) for _, m in parts if m.kind in ("attention", "head_attention", "latent_attention")})
        for i, m in parts:
            if m.kind == "attention" and m.kv_from is None:
                self.k[i] = torch.zeros((num_pages * PAGE, m.kv_heads * 2 * m.dim), dtype=dtype, device=device)
                self.v[i] = torch.zeros((num_pages * PAGE, m.kv_heads * m.vdim), dtype=dtype, device=device)
            elif m.kind == "head_attention":
                self.k[i] = torch.zeros((num_pages * PAGE, m.kv_heads * m.dim), dtype=dtype, device=device)
                self.v[i] = torch.zeros((num_pages * PAGE, m.kv_heads * m.vdim), dtype=dtype, device=device)
            elif m.kind in ("gla", "hgrn2", "retention"):
                self.state[i] = torch.zeros((num_slots, m.heads, m.dim, m.vdim), dtype=torch.float32, device=device)
            elif m.kind == "latent_attention":
                self.latent[i] = torch.zeros((num_pages * PAGE, m.latent_width), dtype=dtype, device=device)
            elif m.kind == "delta":
                self.state[i] = torch.zeros((num_slots, m.heads, m.dim, m.vdim), dtype=torch.float32, device=device)
                self.conv[i] = torch.zeros((num_slots, m.conv - 1, m.conv_channels), dtype=dtype, device=device)

    @property
    def has_state(self) -> bool:
        return bool(self.state)

    @property
    def shareable(self) -> bool:
        return not self.has_state and not self.window

    def take_slot(self) -> int:
        if not self.has_state:
            return -1
        if not self.free_slots:
            raise MemoryError("no free recurrent-state slot")
        return self.free_slots.pop()

    def give_slot(self, slot: int):
        if slot >= 0:
            self.free_slots.append(slot)

    def first_live_page(self, pos: int) -> int:
        """The first page, kept ones aside, that a query at position ``pos`` or later can still look at."""
        return min(first_key(pos, *m) for m in self.looks_back) // PAGE if self.window else 0

    def pages_needed(self, tokens: int) -> int:
        """The most pages a sequence of ``tokens`` tokens holds at a time."""
        n = (tokens + PAGE - 1) // PAGE
        return min(n, (self.window - 1) // PAGE + 2 + self.kept_pages) if self.window else n

    def bytes_per_token(self) -> float:
        return float(sum(t.shape[1] * t.element_size() for d in (self.k, self.v, self.latent) for t in d.values()))

    def bytes_per_sequence(self) -> float:
        """Recurrent state of one sequence, whatever its length."""
        return float(sum(t[0].numel() * t.element_size() for d in (self.state, self.conv) for t in d.values())) if self.num_slots else 0.0
