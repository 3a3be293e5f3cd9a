"""Decoders built from a list of layers with different sequence mixers: the mixers and the feed-forwards as parameter modules
with one forward pass each over a batch description (``StepBatch``), and the model that runs them over a 32-bit residual
stream, or over several (``StreamResidual``).  Where the norms stand is the layer class's business: before and after every sublayer
(``SandwichLayer``), on its output only (``OutputNormLayer``), before it (``StreamLayer``).

The engine drives the same passes for prompts, for portions of prompts and for decoding; what is remembered between steps
lives in ``inference.mixer_cache``.  A pass of one layer is, for a prompt or a decode step alike:

  attention   GEMM [q | k | v], rotation + cache append, attention with its epilogue (difference of the maps, norm, scale), GEMM
  head_attention  GEMM [q | k | v | gates], head norms + rotation + cache append, attention with its epilogue (sink, gates), GEMM
  latent      GEMM [q | latent | gates], norm of the latent + cache append, then
                prompts   GEMM latent -> [k | v], attention with the head gates in its epilogue, GEMM
                decoding  queries taken to the latent space, attention over the cached latents, values read out of the result
                          head by head with the gates, GEMM
  delta       GEMM [q | k | v | gate | b | a], convolution + unit lengths + gates, recurrence (+ gated norm), GEMM
  gla         GEMM [q | k | v | gate | a1], decays + products of four tokens, recurrence, gated norm (decoding: one kernel), GEMM
  hgrn2       GEMM [q | f | v], forget gates + products of four tokens, recurrence, norm (decoding: one kernel), GEMM
  pair        GEMM [left | right], then on its columns the steps of head_attention and of
                retention  rotation + products of four tokens, recurrence, gated norm (decoding: one kernel), GEMM
  MLP         GEMM [gate | up], act(gate) * up, GEMM;  or GEMM with the squared relu in its epilogue, GEMM
  mixture     router GEMM (fp32 logits), top-k + expert segments, rows by expert, grouped GEMM, silu(gate) * up, grouped GEMM,
              weighted sum + (gated) shared expert
  between     norm and scale of the sublayer's output (or the sum of two), residual add (or the mixing of the streams) and norm of (or
              rounding for) the next sublayer, one kernel

bf16 parameters: bf16 activations and tensor-core products; fp32 parameters: everything in true fp32."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn as nn

from ..ops import functional as F
from ..ops import moe as X
from ..ops import stack as K


@dataclass
class StepBatch:
    """B sequences with S rows each (rows past a sequence's length are padding).  ``decode``: one token per sequence over the
    cache.  Otherwise a prompt (``pos0`` = 0) or, for one sequence, the portion that starts at ``pos0``."""
    tokens: torch.Tensor                       # [B*S] int64
    positions: torch.Tensor                    # [B*S] int32
    B: int
    S: int
    slots: Optional[torch.Tensor] = None       # [B*S] int64 flat cache slots, -1: not cached
    state_slots: Optional[torch.Tensor] = None # [B] int32
    lens: Optional[torch.Tensor] = None        # [B] int32, None: S
    pos0: int = 0
    pages: Optional[torch.Tensor] = None       # int32, the page list of the sequence (pos0 > 0)
    block_table: Optional[torch.Tensor] = None # [B, max_pages] int32 (decode)
    decode: bool = False


def _param(*shape, device, dtype, pitched=True):
    w = K.padded_weight(*shape[-2:], dtype, device, shape[:-2]) if pitched and len(shape) > 1 else torch.zeros(shape, dtype=dtype, device=device)
    return nn.Parameter(w, requires_grad=False)


class Sublayer(nn.Module):
    """A mixer or feed-forward of layer ``index`` (its cache) with the tensors of layer ``source``."""

    def __init__(self, index: int):
        super().__init__()
        self.index = self.source = index

    def finalize(self):
        pass

    def at(self, index: int):
        """The same tensors as a part of another layer."""
        m = copy.copy(self)
        m.index = index
        return m


class DiffAttention(Sublayer):
    """Differential attention with an optional window and optional keys / values of an earlier layer."""
    linear_names = ("qkv", "o")

    def __init__(self, spec, hidden: int, eps: float, index: int, device, dtype):
        super().__init__(index)
        self.spec, self.eps = spec, eps
        self.nq = 2 * spec.heads
        self.nk = 0 if spec.kv_from is not None else 2 * spec.kv_heads
        self.v_cols = spec.kv_heads * spec.vdim if self.nk else 0
        kw = dict(device=device, dtype=dtype)
        self.qkv = _param((self.nq + self.nk) * spec.dim + self.v_cols, hidden, **kw)
        self.o = _param(hidden, spec.heads * spec.vdim, **kw)
        for n in ("lq1", "lk1", "lq2", "lk2"):
            setattr(self, n, _param(spec.dim, **kw))
        self._lambda = None

    def tensors(self):
        s, a = self.spec, self.nq * self.spec.dim
        b = a + self.nk * s.dim
        yield "q", self.qkv.data[:a]
        if self.nk:
            yield "k", self.qkv.data[a:b]
            yield "v", self.qkv.data[b:]
        for n in ("lq1", "lk1", "lq2", "lk2", "o"):
            yield n, getattr(self, n).data

    def finalize(self):
        d = lambda n: getattr(self, n).data.double()
        self._lambda = float(torch.exp((d("lq1") * d("lk1")).sum()) - torch.exp((d("lq2") * d("lk2")).sum()) + self.spec.diff)

    def forward(self, h, b: StepBatch, cache, rope, lin, kv):
        s = self.spec
        if self._lambda is None:
            self.finalize()
        qkv = lin(h, self.source, "qkv", self.qkv)
        pool = self.index if self.nk else s.kv_from
        K.rope_append(qkv, rope(s.rot), b.positions, self.nq, self.nk, s.dim, s.rot.dims, self.v_cols, b.slots if self.nk else None,
                      cache.k[pool] if self.nk else None, cache.v[pool] if self.nk else None)
        q = qkv[:, :self.nq * s.dim]
        args = (s.heads, s.kv_heads, s.dim, s.vdim, s.window, s.scale, self._lambda, 1.0 - s.diff, self.eps)
        if b.decode:
            o = K.diff_decode(q, cache.k[pool], cache.v[pool], b.block_table, b.positions, *args)
        else:
            if self.nk:                        # keys and values of this step, for this layer and for those that share them
                if b.pos0 == 0:
                    c = self.nq * s.dim
                    kv[self.index] = (qkv[:, c:c + self.nk * s.dim], qkv[:, c + self.nk * s.dim:], b.S)
                else:
                    lo = max(0, b.pos0 - cache.window + 1) if cache.window else 0
                    n = b.pos0 + b.S - lo
                    kv[self.index] = (K.gather_rows(cache.k[pool], b.pages, lo, n), K.gather_rows(cache.v[pool], b.pages, lo, n), n)
            k, v, n = kv[pool]
            o = K.diff_attn(q, k, v, b.B, b.S, n, *args)
        return lin(o, self.source, "o", self.o)


class HeadAttention(Sublayer):
    """Softmax attention with the options of its spec (see ``HeadAttentionSpec``).  ``proj``, ``proj_bias``: rows of another module's
    projection and bias that are this one's (``mix`` then gets its columns of the product)."""
    linear_names = ("proj", "o")

    def __init__(self, spec, hidden: int, eps: float, index: int, device, dtype, proj=None, proj_bias=None):
        super().__init__(index)
        self.spec, self.eps = spec, eps
        kw = dict(device=device, dtype=dtype)
        self.nq, self.nk, self.nv, self.no = spec.heads * spec.dim, spec.kv_heads * spec.dim, spec.kv_heads * spec.vdim, spec.heads * spec.vdim
        n = self.columns(spec)
        self.proj = _param(n, hidden, **kw) if proj is None else proj
        self.proj_bias = proj_bias if proj is not None else _param(n, **kw) if spec.bias else None
        self.o = _param(hidden, self.no, **kw)
        if spec.qk_norm and spec.qk_weight:
            self.q_norm, self.k_norm = _param(spec.dim, **kw), _param(spec.dim, **kw)
        self.temp = _param(spec.heads, **kw) if spec.head_temp else None
        self.sink = _param(spec.heads, **kw) if spec.head_sink else None
        self.options = K.HeadOptions(spec.window, spec.keep_first, spec.softcap, spec.sink, spec.temp_coef, spec.temp_every, spec.chunk)

    @staticmethod
    def columns(spec) -> int:
        return spec.heads * spec.dim + spec.kv_heads * (spec.dim + spec.vdim) + (spec.heads * spec.vdim if spec.gate else 0)

    def tensors(self):
        a, b, c = self.nq, self.nq + self.nk, self.nq + self.nk + self.nv
        for n, lo, hi in (("q", 0, a), ("k", a, b), ("v", b, c)):
            yield n, self.proj.data[lo:hi]
            if self.spec.bias:
                yield n + ".b", self.proj_bias.data[lo:hi]
        if self.spec.gate:
            yield "g", self.proj.data[c:]
        if self.spec.qk_norm and self.spec.qk_weight:
            yield "q.norm", self.q_norm.data
            yield "k.norm", self.k_norm.data
        for n in ("temp", "sink"):
            if getattr(self, n) is not None:
                yield n, getattr(self, n).data
        yield "o", self.o.data

    def _past(self, cache, b):
        """Keys and values that the portion from b.pos0 on looks at: the kept first tokens and the window (or chunk) of its first query, or
        the whole sequence, this portion's included."""
        s, n = self.spec, b.pos0 + b.S
        lo = 0 if s.chunk and s.keep_first else self.options.first_key(b.pos0)
        kept = min(s.keep_first, lo)
        out = []
        for pool in (cache.k[self.index], cache.v[self.index]):
            t = K.gather_rows(pool, b.pages, lo, n - lo)
            out.append(torch.cat([K.gather_rows(pool, b.pages, 0, kept), t]) if kept else t)
        return out[0], out[1], kept + n - lo

    def mix(self, p, b: StepBatch, cache, rope):
        """The heads' outputs, of the projected rows p."""
        s, i = self.spec, self.index
        norms = ((self.q_norm.data, self.k_norm.data) if s.qk_weight else (None, None)) + (self.eps,) if s.qk_norm else None
        K.rope_append(p, rope(s.rot), b.positions, s.heads, s.kv_heads, s.dim, s.rot.dims if s.rot else 0, self.nv, b.slots, cache.k[i], cache.v[i],
                      norms, self.temp.data if self.temp is not None else None)
        c = self.nq + self.nk
        q, gate = p[:, :self.nq], p[:, c + self.nv:c + self.nv + self.no] if s.gate else None
        sizes, sinks = (s.heads, s.kv_heads, s.dim, s.vdim, s.scale, gate, self.options), self.sink.data if self.sink is not None else None
        if b.decode:
            return K.head_decode(q, cache.k[i], cache.v[i], b.block_table, b.positions, *sizes, sinks=sinks)
        k, v, n = self._past(cache, b) if b.pos0 else (p[:, self.nq:c], p[:, c:c + self.nv], b.S)
        return K.head_attn(q, k, v, b.B, b.S, n, *sizes, b.pos0, sinks)

    def forward(self, h, b: StepBatch, cache, rope, lin, kv):
        bias = {"bias": self.proj_bias.data} if self.proj_bias is not None else {}
        return lin(self.mix(lin(h, self.source, "proj", self.proj, **bias), b, cache, rope), self.source, "o", self.o)


class GatedDelta(Sublayer):
    """Gated delta rule with a short convolution in front and a gated norm behind."""
    linear_names = ("proj", "o")

    def __init__(self, spec, hidden: int, eps: float, index: int, device, dtype):
        super().__init__(index)
        self.spec, self.eps = spec, eps
        kw = dict(device=device, dtype=dtype)
        self.hv = spec.heads * spec.vdim
        self.proj = _param(spec.conv_channels + self.hv + 2 * spec.heads, hidden, **kw)
        self.conv = _param(spec.conv_channels, spec.conv, pitched=False, **kw)
        self.A_log, self.dt_bias, self.norm = _param(spec.heads, **kw), _param(spec.heads, **kw), _param(spec.vdim, **kw)
        self.o = _param(hidden, self.hv, **kw)

    def tensors(self):
        s = self.spec
        gd, c = s.kv_heads * s.dim, s.conv_channels
        cuts = {"q": (0, gd), "k": (gd, 2 * gd), "v": (2 * gd, c), "g": (c, c + self.hv),
                "b": (c + self.hv, c + self.hv + s.heads), "a": (c + self.hv + s.heads, c + self.hv + 2 * s.heads)}
        for n, (lo, hi) in cuts.items():
            yield n, self.proj.data[lo:hi]
            if n in ("q", "k", "v"):
                yield n + ".conv", self.conv.data[lo:hi]
        for n in ("A_log", "dt_bias", "norm", "o"):
            yield n, getattr(self, n).data

    def forward(self, h, b: StepBatch, cache, rope, lin, kv):
        s, i = self.spec, self.index
        G, H, D, V = s.kv_heads, s.heads, s.dim, s.vdim
        p = lin(h, self.source, "proj", self.proj)
        past = b.decode or b.pos0 > 0
        prep = K.delta_prep(p, self.conv.data, cache.conv[i], b.state_slots, self.A_log.data, self.dt_bias.data, b.lens, b.B, b.S, G, H, D, V, past, b.decode)
        gate = p[:, s.conv_channels:s.conv_channels + self.hv]
        if b.decode:
            o = K.delta_step(prep, cache.state[i], b.state_slots, gate, self.norm.data, self.eps, b.B, G, H, D, V)
        else:
            o = K.gated_norm(K.delta_scan(prep, cache.state[i], b.state_slots, b.lens, b.B, b.S, G, H, D, V, past), gate, self.norm.data, self.eps)
        return lin(o, self.source, "o", self.o)


class GatedLinear(Sublayer):
    """Gated linear attention with a decay per key channel and a gated norm behind."""
    linear_names = ("proj", "o")

    def __init__(self, spec, hidden: int, eps: float, index: int, device, dtype):
        super().__init__(index)
        self.spec, self.eps = spec, eps
        kw = dict(device=device, dtype=dtype)
        self.hd, self.hv = spec.heads * spec.dim, spec.heads * spec.vdim
        self.proj = _param(2 * self.hd + 2 * self.hv + spec.rank, hidden, **kw)
        self.a2, self.a2_b, self.norm = _param(self.hd, spec.rank, **kw), _param(self.hd, **kw), _param(spec.vdim, **kw)
        self.o = _param(hidden, self.hv, **kw)

    def tensors(self):
        at = 0
        for n, width in (("q", self.hd), ("k", self.hd), ("v", self.hv), ("g", self.hv), ("a1", self.spec.rank)):
            yield n, self.proj.data[at:at + width]
            at += width
        yield "a2", self.a2.data
        yield "a2.b", self.a2_b.data
        yield "norm", self.norm.data
        yield "o", self.o.data

    def forward(self, h, b: StepBatch, cache, rope, lin, kv):
        s, state = self.spec, cache.state[self.index]
        p = lin(h, self.source, "proj", self.proj)
        low, sizes = (p, self.a2.data, self.a2_b.data, s.tau), (s.heads, s.dim, s.vdim)
        if b.decode:
            o = K.gla_step(*low, state, b.state_slots, self.norm.data, self.eps, b.B, *sizes)
        else:
            r = K.gla_prep(*low, b.lens, b.B, b.S, *sizes)
            o = K.gla_scan(r, state, b.state_slots, b.lens, b.B, b.S, *sizes, b.pos0 > 0)
            o = K.gated_norm(o, p[:, 2 * self.hd + self.hv:2 * (self.hd + self.hv)], self.norm.data, self.eps)
        return lin(o, self.source, "o", self.o)


class ForgetLinear(Sublayer):
    """Linear attention whose forget gate also decides what is written (HGRN2), with a norm of the heads behind."""
    linear_names = ("proj", "o")

    def __init__(self, spec, hidden: int, eps: float, index: int, device, dtype):
        super().__init__(index)
        self.spec, self.eps = spec, eps
        kw = dict(device=device, dtype=dtype)
        self.hd, self.hv = spec.heads * spec.dim, spec.heads * spec.vdim
        self.proj = _param(2 * self.hd + self.hv, hidden, **kw)
        self.f_b, self.lower, self.norm = _param(self.hd, **kw), _param(self.hd, **kw), _param(spec.vdim, **kw)
        self.o = _param(hidden, self.hv, **kw)

    def tensors(self):
        yield "q", self.proj.data[:self.hd]
        yield "f", self.proj.data[self.hd:2 * self.hd]
        yield "f.b", self.f_b.data
        yield "lower", self.lower.data
        yield "v", self.proj.data[2 * self.hd:]
        yield "norm", self.norm.data
        yield "o", self.o.data

    def forward(self, h, b: StepBatch, cache, rope, lin, kv):
        s, state = self.spec, cache.state[self.index]
        p = lin(h, self.source, "proj", self.proj)
        gates, sizes = (self.f_b.data, self.lower.data), (s.heads, s.dim, s.vdim)
        if b.decode:
            o = K.forget_step(p, *gates, state, b.state_slots, self.norm.data, self.eps, b.B, *sizes)
        else:
            r = K.forget_prep(p, *gates, b.lens, b.B, b.S, *sizes)
            o = K.gated_norm(K.gla_scan(r, state, b.state_slots, b.lens, b.B, b.S, *sizes, b.pos0 > 0), None, self.norm.data, self.eps, p.dtype)
        return lin(o, self.source, "o", self.o)


class Retention(Sublayer):
    """Retention: a fixed decay per head, rotated queries and keys, a norm of the heads without a weight, a gate.  ``proj``: as in
    ``HeadAttention``."""
    linear_names = ("proj", "o")

    def __init__(self, spec, hidden: int, eps: float, index: int, device, dtype, proj=None, proj_bias=None):
        super().__init__(index)
        self.spec, self.eps = spec, eps
        self.hd, self.hv = spec.heads * spec.dim, spec.heads * spec.vdim
        self.proj = _param(self.columns(spec), hidden, device=device, dtype=dtype) if proj is None else proj
        self.o = _param(hidden, self.hv, device=device, dtype=dtype)
        self.decay = torch.tensor(spec.decay, dtype=torch.float32, device=device)

    @staticmethod
    def columns(spec) -> int:
        return 2 * spec.heads * (spec.dim + spec.vdim)

    def tensors(self):
        at = 0
        for n, width in (("q", self.hd), ("k", self.hd), ("v", self.hv), ("g", self.hv)):
            yield n, self.proj.data[at:at + width]
            at += width
        yield "o", self.o.data

    def mix(self, p, b: StepBatch, cache, rope):
        s, state = self.spec, cache.state[self.index]
        turn, sizes = (self.decay, rope(s.rot), s.rot.dims if s.rot else 0, b.positions), (s.heads, s.dim, s.vdim)
        if b.decode:
            return K.retention_step(p, *turn, state, b.state_slots, None, self.eps, b.B, *sizes)
        r = K.retention_prep(p, *turn, b.lens, b.B, b.S, *sizes)
        o = K.gla_scan(r, state, b.state_slots, b.lens, b.B, b.S, *sizes, b.pos0 > 0)
        return K.gated_norm(o, p[:, 2 * self.hd + self.hv:2 * (self.hd + self.hv)], None, self.eps)

    def forward(self, h, b: StepBatch, cache, rope, lin, kv):
        return lin(self.mix(lin(h, self.source, "proj", self.proj), b, cache, rope), self.source, "o", self.o)


class MixerPair(Sublayer):
    """Two mixers on the same input, with one product for the projections of both; returns their two outputs (the layer norms and adds
    them, with the weights ``left_out`` and ``right_out``)."""
    linear_names = ("proj", "left_o", "right_o")

    def __init__(self, spec, hidden: int, eps: float, index: int, device, dtype):
        super().__init__(index)
        self.spec = spec
        kw = dict(device=device, dtype=dtype)
        kinds = [MIXERS[m.kind] for m in (spec.left, spec.right)]
        self.cut = kinds[0].columns(spec.left)
        n = self.cut + kinds[1].columns(spec.right)
        self.proj = _param(n, hidden, **kw)
        self.proj_bias = _param(n, **kw) if any(getattr(m, "bias", False) for m in (spec.left, spec.right)) else None     # zeros where one has none
        part = lambda t, s: None if t is None else t.data[s]
        self.left, self.right = (c(m, hidden, eps, index, device, dtype, self.proj.data[s], part(self.proj_bias, s))
                                 for c, m, s in zip(kinds, (spec.left, spec.right), (slice(None, self.cut), slice(self.cut, None))))
        self.left_out, self.right_out = _param(hidden, **kw), _param(hidden, **kw)

    left_o = property(lambda self: self.left.o)
    right_o = property(lambda self: self.right.o)

    def finalize(self):
        self.left.finalize()
        self.right.finalize()

    def at(self, index: int):
        m = super().at(index)
        m._modules = dict(self._modules, left=self.left.at(index), right=self.right.at(index))
        return m

    def tensors(self):
        for side in ("left", "right"):
            for n, t in getattr(self, side).tensors():
                yield f"{side}.{n}", t
        yield "left.out", self.left_out.data
        yield "right.out", self.right_out.data

    def forward(self, h, b: StepBatch, cache, rope, lin, kv):
        p = lin(h, self.source, "proj", self.proj, **({"bias": self.proj_bias.data} if self.proj_bias is not None else {}))
        left = lin(self.left.mix(p[:, :self.cut], b, cache, rope), self.source, "left_o", self.left_o)
        return left, lin(self.right.mix(p[:, self.cut:], b, cache, rope), self.source, "right_o", self.right_o)


class LatentAttention(Sublayer):
    """Attention without positions over one cached latent per token, with an output gate per head."""
    linear_names = ("proj", "o")

    def __init__(self, spec, hidden: int, eps: float, index: int, device, dtype):
        super().__init__(index)
        self.spec, self.eps = spec, eps
        kw = dict(device=device, dtype=dtype)
        self.nq, self.nv = spec.heads * spec.dim, spec.heads * spec.vdim
        self.proj = _param(self.nq + spec.kv_rank + spec.heads, hidden, **kw)
        self.norm = _param(spec.kv_rank, **kw)
        self.ukv = _param(self.nq + self.nv, spec.kv_rank, **kw)
        self.o = _param(hidden, self.nv, **kw)

    def tensors(self):
        a = self.nq + self.spec.kv_rank
        yield "q", self.proj.data[:self.nq]
        yield "dkv", self.proj.data[self.nq:a]
        yield "dkv.norm", self.norm.data
        yield "uk", self.ukv.data[:self.nq]
        yield "uv", self.ukv.data[self.nq:]
        yield "g", self.proj.data[a:]
        yield "o", self.o.data

    def forward(self, h, b: StepBatch, cache, rope, lin, kv):
        s, i = self.spec, self.index
        p = lin(h, self.source, "proj", self.proj)
        q, gate = p[:, :self.nq], p[:, self.nq + s.kv_rank:]
        pool = cache.latent[i]
        c = K.latent_append(p[:, self.nq:self.nq + s.kv_rank], self.norm.data, self.eps, b.slots, pool, want_rows=not b.decode and b.pos0 == 0)
        if b.decode:
            u = K.head_linear(q, self.ukv.data[:self.nq], s.heads, s.dim, s.kv_rank, transposed=True)
            u = K.latent_decode(u, pool, b.block_table, b.positions, s.heads, s.kv_rank, s.scale)
            o = K.head_linear(u, self.ukv.data[self.nq:], s.heads, s.kv_rank, s.vdim, gate=gate)
        else:
            n = b.S
            if b.pos0:                         # the latents of the whole sequence so far, this portion's included
                n = b.pos0 + b.S
                c = K.gather_rows(pool, b.pages, 0, n)[:, :s.kv_rank]
            e = lin(c, self.source, "ukv", self.ukv)
            o = K.head_attn(q, e[:, :self.nq], e[:, self.nq:], b.B, b.S, n, s.heads, s.heads, s.dim, s.vdim, s.scale, gate)
        return lin(o, self.source, "o", self.o)


class GatedMLP(Sublayer):
    linear_names = ("gate_up", "down")
    act, limit = "silu", 0.0

    def __init__(self, hidden: int, ff: int, index: int, device, dtype, act=None, limit: float = 0.0):
        super().__init__(index)
        self.ff = ff
        if act:
            self.act, self.limit = act, limit
        self.gate_up = _param(2 * ff, hidden, device=device, dtype=dtype)
        self.down = _param(hidden, ff, device=device, dtype=dtype)

    def tensors(self):
        yield "gate", self.gate_up.data[:self.ff]
        yield "up", self.gate_up.data[self.ff:]
        yield "down", self.down.data

    def forward(self, h, lin):
        return lin(K.glu(lin(h, self.source, "gate_up", self.gate_up), self.act, self.limit), self.source, "down", self.down)


class GeluMLP(GatedMLP):
    act = "gelu_tanh"


class SquaredMLP(Sublayer):
    """down(relu(up h)^2)."""
    linear_names = ("up", "down")

    def __init__(self, hidden: int, ff: int, index: int, device, dtype):
        super().__init__(index)
        self.up, self.down = _param(ff, hidden, device=device, dtype=dtype), _param(hidden, ff, device=device, dtype=dtype)

    def tensors(self):
        yield "up", self.up.data
        yield "down", self.down.data

    def forward(self, h, lin):
        return lin(lin(h, self.source, "up", self.up, act="relu2"), self.source, "down", self.down)


class MixtureMLP(Sublayer):
    """Gated experts chosen per token, and a gated expert that every token runs (with ``shared_gate`` times the sigmoid of one more
    row of the router's matrix)."""

    def __init__(self, hidden: int, spec, index: int, device, dtype):
        super().__init__(index)
        self.spec = spec
        kw = dict(device=device, dtype=dtype)
        self.router = _param(spec.experts + int(spec.shared_gate), hidden, **kw)
        self.router_bias = _param(spec.experts, **kw) if spec.score == "softmax" else None
        self.gate_up, self.down = _param(spec.experts, 2 * spec.ff, hidden, **kw), _param(spec.experts, hidden, spec.ff, **kw)
        self.shared = GatedMLP(hidden, spec.shared_ff, index, device, dtype, spec.act, spec.shared_limit) if spec.shared_ff else None

    def tensors(self):
        F = self.spec.ff
        for e in range(self.spec.experts):
            yield f"e{e}.gate", self.gate_up.data[e, :F]
            yield f"e{e}.up", self.gate_up.data[e, F:]
            yield f"e{e}.down", self.down.data[e]
        yield "router", self.router.data[:self.spec.experts]
        if self.router_bias is not None:
            yield "router.b", self.router_bias.data
        if self.shared is not None:
            for n, t in self.shared.tensors():
                yield "shared." + n, t
        if self.spec.shared_gate:
            yield "shared.sg", self.router.data[self.spec.experts:]

    def forward(self, h, lin):
        s, E = self.spec, self.spec.experts
        z = K.linear(h, self.router.data, out_dtype=torch.float32)
        r = X.route(z[:, :E], self.router_bias.data if self.router_bias is not None else None, s.top, s.score, s.groups, s.keep, s.scale)
        g = X.expert_linear(X.expert_rows(h, r), self.gate_up.data, r)
        y = X.expert_linear(X.expert_glu(g, r, s.act, s.limit), self.down.data, r)
        return X.weighted_sum(y, r, self.shared(h, lin) if self.shared is not None else None, z[:, E:] if s.shared_gate else None)


MIXERS = {"attention": DiffAttention, "delta": GatedDelta, "latent_attention": LatentAttention, "head_attention": HeadAttention, "gla": GatedLinear,
          "hgrn2": ForgetLinear, "retention": Retention, "pair": MixerPair}


class ResidualLayer(nn.Module):
    """A mixer and, unless the layer is a mixer alone, a feed-forward.  ``parts`` lists the groups of sublayers that read the same
    input, with what ``K.res_norm`` does to that input (``pre``) and to their outputs (``post``)."""
    norm_kind = "rms"
    dense_mlp = GatedMLP

    def __init__(self, spec, cfg, index: int, device, dtype):
        super().__init__()
        hidden = cfg.hidden_size
        self.mixer = MIXERS[spec.mixer.kind](spec.mixer, hidden, cfg.norm_eps, index, device, dtype)
        self.mlp = None
        if spec.mixture is not None:
            self.mlp = MixtureMLP(hidden, spec.mixture, index, device, dtype)
        elif spec.ffn_hidden_size:
            self.mlp = self.dense_mlp(hidden, spec.ffn_hidden_size, index, device, dtype)
        for n in self.vector_names():
            setattr(self, n.replace(".", "_"), _param(hidden, device=device, dtype=dtype))

    def vector(self, name):
        return getattr(self, name.replace(".", "_")).data

    def at(self, index: int):
        """The same tensors as another layer, with a cache of its own."""
        l = copy.copy(self)
        l._modules = dict(self._modules, mixer=self.mixer.at(index))
        return l

    @property
    def linears(self):
        """{name: matrix} of the layer's own products (what a low-bit weight format may replace)."""
        out = {}
        if self.mixer.index != self.mixer.source:
            return out
        for m in (self.mixer, self.mlp):
            m = m.shared if isinstance(m, MixtureMLP) else m
            if m is not None:
                out.update({n: getattr(m, n) for n in m.linear_names})
        return out

    def tensors(self):
        for n in self.vector_names():
            yield n, self.vector(n)
        for n, t in self.mixer.tensors():
            yield "mix." + n, t
        if self.mlp is not None:
            for n, t in self.mlp.tensors():
                yield "mlp." + n, t


class SandwichLayer(ResidualLayer):
    """norm1, mixer, norm1b and norm2, feed-forward, norm2b: RMS norms whose weight is the deviation from one."""
    final_names = ("final.norm",)

    def vector_names(self):
        return ("norm1", "norm1b") + (("norm2", "norm2b") if self.mlp is not None else ())

    def parts(self):
        v = self.vector
        yield (self.mixer,), {"w_pre": v("norm1")}, {"w_post": v("norm1b")}
        if self.mlp is not None:
            yield (self.mlp,), {"w_pre": v("norm2")}, {"w_post": v("norm2b")}


class OutputNormLayer(ResidualLayer):
    """The sublayers read the residual itself; a layer norm (norm1, norm2) and a per-channel scale (ls1, ls2) on what they return."""
    norm_kind = "layer"
    dense_mlp = SquaredMLP
    final_names = ("final.norm", "final.norm.b")

    def vector_names(self):
        return sum(((f"norm{k}", f"norm{k}.b", f"ls{k}") for k in ((1, 2) if self.mlp is not None else (1,))), ())

    def parts(self):
        v = self.vector
        for k, m in ((1, self.mixer), (2, self.mlp)):
            if m is not None:
                w = v(f"norm{k}")
                yield (m,), {"cast": w.dtype}, {"w_post": w, "b_post": v(f"norm{k}.b"), "scale_post": v(f"ls{k}")}


class ParallelLayer(ResidualLayer):
    """One RMS norm (norm1), whose output the mixer and the feed-forward both read; their sum goes to the residual as it is."""
    norm_kind = "plain"
    dense_mlp = GeluMLP
    final_names = ("final.norm",)

    def vector_names(self):
        return ("norm1",)

    def parts(self):
        yield (self.mixer,) if self.mlp is None else (self.mixer, self.mlp), {"w_pre": self.vector("norm1")}, {}


class StreamLayer(ResidualLayer):
    """A norm in groups (norm1, norm2) in front of the mixer and the feed-forward, each between a reading (hc<q>.in) and a mixing (hc<q>.mix,
    hc<q>.out) of the residual's streams."""
    norm_kind = "plain"
    final_names = ("final.norm",)

    def __init__(self, spec, cfg, index: int, device, dtype):
        super().__init__(spec, cfg, index, device, dtype)
        self.hc = nn.ModuleList()
        for _ in range(1 if self.mlp is None else 2):
            m = nn.Module()
            m.read, m.write = (_param(cfg.streams, device=device, dtype=dtype) for _ in range(2))
            m.mix = _param(cfg.streams, cfg.streams, device=device, dtype=dtype, pitched=False)
            self.hc.append(m)

    def vector_names(self):
        return ("norm1",) + (("norm2",) if self.mlp is not None else ())

    def tensors(self):
        yield from super().tensors()
        for q, m in enumerate(self.hc, 1):
            for n, t in (("in", m.read), ("out", m.write), ("mix", m.mix)):
                yield f"hc{q}.{n}", t.data

    def parts(self):
        for q, (m, hc) in enumerate(zip((self.mixer, self.mlp), self.hc), 1):
            post = {"mix": hc.mix.data, "out": hc.write.data}
            if isinstance(m, MixerPair):
                post.update(w_post=m.left_out.data, w_post2=m.right_out.data, share=0.5)
            yield (m,), {"w_pre": self.vector(f"norm{q}"), "w_in": hc.read.data}, post


def _plain_linear(x, index, name, w, act=None, bias=None):
    return K.linear(x, w.data, act=act, bias=bias)


class StackModel(nn.Module):
    """Embedding, layers, final norm, head.  ``run`` is the pass the engine drives; ``forward`` / ``hidden_states`` are whole
    sequences without a cache."""
    kernel_units = K.UNITS
    layer_cls = SandwichLayer
    embed_norm_name = None       # a norm between the embedding and the residual
    linear, activation = staticmethod(K.linear), staticmethod(K.activation)
    runs_fp32 = True             # every kernel of the pass has a true fp32 form

    def __init__(self, cfg, device=None, dtype=torch.bfloat16, seed: Optional[int] = 0):
        super().__init__()
        self.cfg = cfg
        device = torch.device(device if device is not None else "cpu")
        kw = dict(device=device, dtype=dtype)
        self.tok_embeddings = _param(cfg.vocab_size, cfg.hidden_size, **kw)
        own = {i: self.layer_cls(l, cfg, i, device, dtype) for i, l in enumerate(cfg.layers) if l.weights_of is None}
        self.layers = nn.ModuleList([own[i] if i in own else own[l.weights_of].at(i) for i, l in enumerate(cfg.layers)])
        self.embed_norm = _param(cfg.hidden_size, **kw) if self.embed_norm_name else None
        self.norm = _param(cfg.hidden_size, **kw)
        self.norm_bias = _param(cfg.hidden_size, **kw) if len(self.layer_cls.final_names) > 1 else None
        self.lm_head = self.tok_embeddings if cfg.tie_embeddings else _param(cfg.vocab_size, cfg.hidden_size, **kw)
        self._rope = {}
        if seed is not None:
            self.init_weights(seed)

    def init_weights(self, seed: int = 0):
        """Random weights that keep activations of order one: N(0, 1 / fan-in) matrices, small deviations for the norms, decays
        between about 0.5 and 1, streams that go on with a part of one another."""
        about_one = lambda n: n.endswith(("mix.norm", "dkv.norm", ".temp", "left.out", "right.out")) or \
            (self.layer_cls.norm_kind != "rms" and n.rsplit(".", 1)[-1] in ("norm", "norm1", "norm2", "ls1", "ls2"))
        g = torch.Generator(device="cpu").manual_seed(seed)
        with torch.no_grad():
            for name, t in self.named_tensors():
                leaf = name.rsplit(".", 1)[-1]
                r = torch.randn(t.shape, generator=g)
                if leaf == "A_log":
                    r = r * 0.5 - 1.5
                elif leaf == "conv":
                    r = r * t.shape[1] ** -0.5
                elif ".hc" in name:
                    r = (torch.eye(t.shape[0]) * 0.8 if leaf == "mix" else 1 / t.shape[0] if leaf == "in" else 1) + 0.2 * r
                elif leaf == "lower":
                    r = torch.sigmoid(r)
                elif t.dim() == 2:
                    r = r * (1.0 if name == self.embed_name else t.shape[1] ** -0.5)
                elif about_one(name):
                    r = 1 + 0.1 * r
                else:
                    r = 0.1 * r
                t.copy_(r.to(t.dtype))
        self.finalize()

    def finalize(self):
        """Derived constants, after the parameters have changed."""
        for l in self.layers:
            l.mixer.finalize()

    embed_name, head_name = "embed", "head"

    def named_tensors(self):
        """(name in the model folder, view into the parameters) pairs."""
        out = [(self.embed_name, self.tok_embeddings.data)]
        if self.embed_norm is not None:
            out.append((self.embed_norm_name, self.embed_norm.data))
        for i, l in enumerate(self.layers):
            if l.mixer.source == i:
                out += [(f"l{i}.{n}", t) for n, t in l.tensors()]
        out += list(zip(self.layer_cls.final_names, (t.data for t in (self.norm, self.norm_bias) if t is not None)))
        return out if self.cfg.tie_embeddings else out + [(self.head_name, self.lm_head.data)]

    def get_parameters(self):
        return list(self.parameters())

    def param_count(self) -> int:
        return sum(t.numel() for _, t in self.named_tensors())

    def vocab_size(self) -> int:
        return self.cfg.vocab_size

    @property
    def dtype(self):
        return self.tok_embeddings.dtype

    @property
    def device(self):
        return self.tok_embeddings.device

    # ------------------------------------------------------------------ passes
    def rope(self, spec, max_pos: int):
        """cos / sin tables of one rotation for at least ``max_pos`` positions."""
        t = self._rope.get(spec)
        if t is None or t[0].shape[0] < max_pos or t[0].device != self.device:
            mode, factor = ("linear", spec.linear) if spec.yarn_factor is None else ("yarn", spec.yarn_factor)
            t = F.rope_tables(spec.dims, max_pos, spec.base, mode, factor, spec.yarn_original, 1.0, spec.yarn_fast, spec.yarn_slow,
                              device=self.device, yarn_ramp_max=spec.dims - 1)
            self._rope[spec] = t
        return t

    def make_cache(self, num_pages: int, num_slots: int):
        from ..inference.mixer_cache import MixerCache
        return MixerCache(self.cfg, num_pages, num_slots, self.dtype, self.device)

    def new_residual(self, n: int):
        return torch.empty((n, self.cfg.hidden_size), dtype=torch.float32, device=self.device)

    def between(self, x, **kw):
        """What stands between two groups of sublayers (see ``parts`` of the layer classes)."""
        return K.res_norm(x, self.cfg.norm_eps, kind=self.layer_cls.norm_kind, **kw)

    def first(self, x, b, pre):
        return self.between(x, ids=b.tokens, table=self.tok_embeddings.data, scale=self.cfg.embedding_scale,
                            w_post=self.embed_norm.data if self.embed_norm is not None else None, **pre)

    def last_norm(self):
        return {"w_pre": self.norm.data, "b_pre": self.norm_bias.data if self.norm_bias is not None else None}

    def run(self, b: StepBatch, cache, max_pos: int, row_index=None, lin=_plain_linear, residuals=None):
        """One step over all layers.  Returns the final-normed rows (of ``row_index``, int32; all rows without it).
        ``residuals``: a list that receives a copy of the residual stream after every layer."""
        x = self.new_residual(b.tokens.shape[0])
        rope = lambda spec: self.rope(spec, max_pos) if spec is not None else None
        parts = [(i, l) + p for i, l in enumerate(self.layers) for p in l.parts()]
        pre = [p[3] for p in parts] + [self.last_norm()]
        h = self.first(x, b, pre[0])
        kv = {}
        for k, (i, l, group, _, post) in enumerate(parts):
            ys = ()
            for m in group:
                y = m(h, b, cache, rope, lin, kv) if m is l.mixer else m(h, lin)
                ys += y if isinstance(y, tuple) else (y,)
            post = dict(post, y=ys[0], y2=ys[1] if len(ys) > 1 else None)
            last = k + 1 == len(parts)
            if residuals is not None and (last or parts[k + 1][0] != i):
                z = x.clone()
                self.between(z, **post)
                residuals.append(z if z.dim() == 2 else z.sum(1))
            h = self.between(x, row_index=row_index if last else None, **post, **pre[k + 1])
        return h

    def head(self, h):
        """fp32 logits of final-normed rows."""
        return K.linear(h, self.lm_head.data, out_dtype=torch.float32)

    @torch.no_grad()
    def hidden_states(self, ids, residuals=None):
        """Final-normed rows [B*S, H] of whole sequences ids [B, S]."""
        B, S = ids.shape
        dev = self.device
        b = StepBatch(ids.reshape(-1).to(dev), torch.arange(S, dtype=torch.int32, device=dev).repeat(B), B, S,
                      state_slots=torch.arange(B, dtype=torch.int32, device=dev))
        return self.run(b, self.make_cache(0, B), S, residuals=residuals)

    @torch.no_grad()
    def forward(self, ids):
        return self.head(self.hidden_states(ids)).view(*ids.shape, -1)


class StreamResidual:
    """For a ``StackModel`` whose residual is ``cfg.streams`` hyper-connected streams (with ``StreamLayer``), normed in groups."""

    def new_residual(self, n: int):
        return torch.empty((n, self.cfg.streams, self.cfg.hidden_size), dtype=torch.float32, device=self.device)

    def between(self, x, **kw):
        return K.stream_norm(x, self.cfg.norm_eps, groups=self.cfg.norm_groups, **kw)

    def first(self, x, b, pre):
        return self.between(x, ids=b.tokens, table=self.tok_embeddings.data, scale=self.cfg.embedding_scale, **pre)

    def last_norm(self):
        return {"w_pre": self.norm.data}         # of the sum of the streams
