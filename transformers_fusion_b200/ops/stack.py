"""Raw operators of decoders that are a stack of different sequence mixers over a 32-bit residual stream: norms around
every sublayer, streams of residuals, partial rotary embedding, differential attention, softmax attention with options, latent attention, gated
delta rule, linear attention with decays (gated, forget-gated, retention), true fp32 products.

As in ``functional``: CUDA tensors go to the sm_100a kernels (``csrc/kernels/stack_ops.cu``, ``streams.cu``, ``diff_attention.cu``, ``head_attention.cu``,
``latent_attention.cu``, ``delta_rule.cu``, ``gated_linear.cu``), CPU tensors run the plain PyTorch statement of the same math.  Activations are bf16 or fp32 (the dtype of
the tensors decides); the residual, norms, rotation, attention scores and weights, and the recurrence are fp32 in both."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import NamedTuple, Optional

import torch

from . import _lib
from . import functional as F
from ._lib import c_f, c_i, c_ll, c_p, check, ptr, stream

UNITS = ("tfb_host", "gemm_bf16", "skinny_linear", "stack_ops", "diff_attention", "delta_rule")    # translation units these operators need
UNITS_LATENT = ("tfb_host", "gemm_bf16", "skinny_linear", "stack_ops", "head_attention", "latent_attention", "moe_serve")
UNITS_GATED = ("tfb_host", "gemm_bf16", "skinny_linear", "stack_ops", "head_attention", "gated_linear", "moe_serve")
UNITS_STREAMS = UNITS_GATED + ("streams",)
PAGE = 16
ACT = {None: 0, "relu2": 4}      # codes of the product epilogues (gemm_bf16.cu: apply_act)
GLU = {"silu": 0, "gelu_tanh": 1, "clamped": 2}      # tfb_elem.cuh: glu_value
NORM = {"rms": 0, "layer": 1, "plain": 2}

_lib.register("tfb_res_norm", [c_p, c_p, c_ll, c_f, c_i, c_p, c_ll, c_p, c_ll, c_p, c_ll, c_p, c_p, c_p, c_p, c_p, c_p, c_ll, c_p, c_i, c_i, c_f, c_i, c_i, c_p])
_lib.register("tfb_stream_norm", [c_p, c_p, c_ll, c_f, c_i, c_p, c_i, c_p, c_ll, c_p, c_ll, c_p, c_p, c_f, c_p, c_p, c_p, c_p, c_i, c_p, c_ll, c_p, c_i, c_i,
                                  c_f, c_i, c_p])
_lib.register("tfb_glu", [c_p, c_ll, c_p, c_ll, c_i, c_i, c_i, c_f, c_i, c_p])
_lib.register("tfb_rope_append", [c_p, c_ll, c_p, c_p, c_i, c_p, c_p, c_p, c_p, c_ll, c_i, c_i, c_i, c_i, c_i, c_i, c_i, c_p])
_lib.register("tfb_norm_rope_append", [c_p, c_ll, c_p, c_p, c_p, c_f, c_p, c_p, c_i, c_p, c_p, c_p, c_p, c_ll, c_i, c_i, c_i, c_i, c_i, c_i, c_i, c_p])
_lib.register("tfb_gather_rows", [c_p, c_ll, c_p, c_i, c_i, c_i, c_p, c_i, c_i, c_p])
_lib.register("tfb_gemm_f32", [c_p, c_ll, c_p, c_ll, c_p, c_ll, c_i, c_i, c_i, c_i, c_p, c_p])
_lib.register("tfb_skinny_fits", [c_i, c_i, c_i])
_lib.register("tfb_skinny_linear", [c_p, c_ll, c_p, c_ll, c_p, c_ll, c_i, c_i, c_i, c_i, c_i, c_i, c_p, c_p])
_lib.register("tfb_act_rows", [c_p, c_ll, c_p, c_ll, c_i, c_i, c_i, c_i, c_p])
_lib.register("tfb_latent_append", [c_p, c_ll, c_p, c_f, c_p, c_p, c_ll, c_p, c_ll, c_i, c_i, c_i, c_i, c_p])
_lib.register("tfb_head_linear", [c_p, c_ll, c_i, c_p, c_ll, c_p, c_ll, c_i, c_i, c_i, c_i, c_i, c_p])
_lib.register("tfb_skinny_linear_heads", [c_p, c_ll, c_i, c_p, c_ll, c_p, c_ll, c_p, c_ll, c_i, c_i, c_i, c_i, c_i, c_p])
_lib.register("tfb_gemm_f32_heads", [c_p, c_ll, c_i, c_p, c_ll, c_i, c_p, c_ll, c_i, c_p, c_ll, c_i, c_i, c_i, c_i, c_p])
_lib.register("tfb_head_attn", [c_p, c_ll, c_p, c_ll, c_p, c_ll, c_p, c_ll, c_p, c_ll, c_i, c_i, c_i, c_i, c_i, c_i, c_i, c_i, c_f, c_i, c_i, c_i, c_f, c_i,
                                c_p, c_f, c_i, c_i, c_i, c_p, c_p])
_lib.register("tfb_head_decode_plan", [c_i, c_i, c_i, c_i, c_i, c_i, c_i])
_lib.register("tfb_head_decode", [c_p, c_ll, c_p, c_p, c_ll, c_p, c_i, c_i, c_p, c_p, c_ll, c_p, c_ll, c_i, c_p, c_p, c_i, c_i, c_i, c_i, c_i, c_i, c_f,
                                  c_i, c_i, c_i, c_f, c_i, c_p, c_f, c_i, c_i, c_p, c_p])
_lib.register("tfb_gla_prep", [c_p, c_ll, c_p, c_ll, c_p, c_i, c_f, c_p] + [c_p] * 5 + [c_i] * 7 + [c_p])
_lib.register("tfb_gla_scan_segments", [c_i] * 5)
_lib.register("tfb_gla_scan", [c_p] * 7 + [c_i, c_p] + [c_i] * 6 + [c_p, c_i, c_p, c_p, c_p])
_lib.register("tfb_gla_step", [c_p, c_ll, c_p, c_ll, c_p, c_i, c_f, c_p, c_p, c_i, c_p, c_p, c_ll, c_i, c_i, c_i, c_i, c_f, c_i, c_p])
_lib.register("tfb_forget_prep", [c_p, c_ll, c_p, c_p, c_p] + [c_p] * 5 + [c_i] * 7 + [c_p])
_lib.register("tfb_forget_step", [c_p, c_ll, c_p, c_p, c_i, c_p, c_p, c_i, c_p, c_p, c_ll, c_i, c_i, c_i, c_i, c_f, c_i, c_p])
_lib.register("tfb_retention_prep", [c_p, c_ll, c_p, c_p, c_p, c_i, c_i, c_p, c_p] + [c_p] * 5 + [c_i] * 7 + [c_p])
_lib.register("tfb_retention_step", [c_p, c_ll, c_p, c_p, c_p, c_i, c_i, c_p, c_i, c_p, c_p, c_i, c_p, c_p, c_ll, c_i, c_i, c_i, c_i, c_f, c_i, c_p])
_lib.register("tfb_latent_decode_plan", [c_i, c_i, c_i, c_i, c_i])
_lib.register("tfb_latent_decode", [c_p, c_ll, c_p, c_ll, c_p, c_i, c_i, c_p, c_p, c_ll, c_p, c_p, c_i, c_i, c_i, c_i, c_i, c_f, c_i, c_p, c_p])
_lib.register("tfb_diff_attn_fwd", [c_p, c_ll, c_p, c_ll, c_p, c_ll, c_p, c_ll, c_i, c_i, c_i, c_i, c_i, c_i, c_i, c_i, c_f, c_f, c_f, c_f, c_i,
                                    c_p, c_p])
_lib.register("tfb_diff_decode_tc", [c_i, c_i, c_i])
_lib.register("tfb_diff_decode", [c_p, c_ll, c_p, c_p, c_ll, c_p, c_i, c_i, c_p, c_p, c_ll, c_p, c_p, c_i, c_i, c_i, c_i, c_i, c_i, c_i, c_f, c_f,
                                  c_f, c_f, c_i, c_p, c_p])
_lib.register("tfb_delta_padded_dim", [c_i])
_lib.register("tfb_delta_prep", [c_p, c_ll, c_p, c_p, c_p, c_i] + [c_p] * 10 + [c_i] * 10 + [c_p])
_lib.register("tfb_delta_scan", [c_p] * 7 + [c_i, c_p] + [c_i] * 7 + [c_p, c_p])
_lib.register("tfb_gated_norm", [c_p, c_p, c_ll, c_p, c_p, c_ll, c_i, c_i, c_i, c_f, c_i, c_p])
_lib.register("tfb_delta_step", [c_p, c_p, c_p, c_p, c_p, c_p, c_p, c_p, c_i, c_p, c_ll, c_p, c_p, c_ll, c_i, c_i, c_i, c_i, c_i, c_i, c_f, c_i, c_p])


def _f32(t) -> int:
    assert t.dtype in (torch.float32, torch.bfloat16), t.dtype
    return int(t.dtype == torch.float32)


def rows(n: int, width: int, dtype, device) -> torch.Tensor:
    """Uninitialised [n, width] activations whose row pitch is a multiple of 8 elements (TMA wants 16-byte pitches)."""
    return torch.empty((n, (width + 7) // 8 * 8), dtype=dtype, device=device)[:, :width]


def padded_weight(n: int, width: int, dtype, device, lead=()) -> torch.Tensor:
    """Zero [*lead, n, width] matrices with the same pitch rule."""
    return torch.zeros((*lead, n, (width + 7) // 8 * 8), dtype=dtype, device=device)[..., :width]


# ---------------------------------------------------------------------------------------------------- products
def linear(x, w, out_dtype=None, act=None, bias=None):
    """act(x [M, K] @ w [N, K]^T + bias [N]).  bf16 operands: tensor-core product with fp32 accumulation (``out_dtype`` fp32 keeps the
    accumulator's precision), in a form of its own for few rows; fp32 operands: FFMA in true fp32.  ``act``: None or "relu2"."""
    out_dtype = out_dtype or x.dtype
    if not x.is_cuda:
        y = x.float() @ w.float().t()
        return activation(y if bias is None else y + bias.float(), act).to(out_dtype)
    M, K = x.shape
    N = w.shape[0]
    out = rows(M, N, out_dtype, x.device)
    assert bias is None or (bias.dtype == x.dtype and bias.shape == (N,) and bias.is_contiguous())
    if x.dtype == torch.float32:
        assert w.dtype == torch.float32 and w.shape[1] == K and x.stride(1) == 1 and w.stride(1) == 1
        check(_lib.lib().tfb_gemm_f32(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0), M, N, K, ACT[act],
                                      ptr(bias), stream()), "gemm_f32")
        return out
    if x.dtype == w.dtype == torch.bfloat16 and x.stride(1) == w.stride(1) == 1 and (x.stride(0) | w.stride(0)) % 8 == 0 and \
            (x.data_ptr() | w.data_ptr()) % 16 == 0 and _lib.lib().tfb_skinny_fits(M, N, K):
        check(_lib.lib().tfb_skinny_linear(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0), M, N, K, ACT[act],
                                           int(out_dtype == torch.float32), 0, ptr(bias), stream()), "skinny_linear")
        return out
    if act is None:
        return F.gemm(x, w, out=out, bias=bias)
    assert x.dtype == w.dtype == torch.bfloat16 and x.stride(1) == w.stride(1) == 1 and out_dtype == torch.bfloat16
    check(_lib.lib().tfb_gemm_bf16(x.data_ptr(), x.stride(0), 0, w.data_ptr(), w.stride(0), 0, out.data_ptr(), out.stride(0), M, N, K, ptr(bias), None, 0,
                                   1.0, ACT[act], 0, 0, _lib.status_word(x.device).data_ptr(), stream()), "gemm_bf16")
    return out


def activation(x, act):
    """The activation of ``linear`` alone."""
    if act is None:
        return x
    assert act == "relu2", act
    if not x.is_cuda:
        return torch.relu(x.float()).square().to(x.dtype)
    out = rows(*x.shape, x.dtype, x.device)
    check(_lib.lib().tfb_act_rows(x.data_ptr(), x.stride(0), out.data_ptr(), out.stride(0), *x.shape, ACT[act], _f32(x), stream()), "act_rows")
    return out


# ---------------------------------------------------------------------------------------------------- norms
def centred_rms(x, w, eps):
    xf = x.float()
    return xf / torch.sqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * (1 + w.float())


def plain_rms(x, w, eps):
    xf = x.float()
    return xf / torch.sqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w.float()


def layer_norm(x, w, b, eps):
    d = x.float()
    d = d - d.mean(-1, keepdim=True)
    return d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + eps) * w.float() + b.float()


def res_norm(x, eps, *, y=None, y2=None, w_post=None, b_post=None, scale_post=None, w_pre=None, b_pre=None, cast=None, ids=None, table=None,
             scale=1.0, row_index=None, dtype=None, kind="rms"):
    """x += norm(y; w_post, b_post) * scale_post + y2 on the fp32 residual ``x`` [n, H] in place (y itself without ``w_post``); returns
    norm(x; w_pre, b_pre) in the activation dtype, x itself in the dtype ``cast`` without ``w_pre``, None without both.  ``kind``:
    "rms" (weights are deviations from one, no bias), "plain" (weights themselves, no bias) or "layer".  ``ids``: x starts as
    scale * table[ids], normed with ``w_post`` if there is no y.  ``row_index`` (int32): only those rows are computed and
    returned, and x keeps its values."""
    if not x.is_cuda:
        norm = {"rms": lambda t, w, b: centred_rms(t, w, eps), "plain": lambda t, w, b: plain_rms(t, w, eps),
                "layer": lambda t, w, b: layer_norm(t, w, b, eps)}[kind]
        v = table[ids.long()].float() * scale if ids is not None else x
        if y is None and w_post is not None:
            v = norm(v, w_post, b_post)
        if y is not None:
            z = y.float() if w_post is None else norm(y, w_post, b_post)
            z = z if scale_post is None else z * scale_post.float()
            v = v + (z if y2 is None else z + y2.float())
        if row_index is None:
            x.copy_(v)
        else:
            v = v[row_index.long()]
        if w_pre is None:
            return None if cast is None else v.to(cast, copy=True)
        return norm(v, w_pre, b_pre).to(dtype or w_pre.dtype)
    H = x.shape[1]
    n = x.shape[0] if row_index is None else row_index.shape[0]
    w = next(t for t in (w_pre, w_post, table, y) if t is not None)
    a = rows(n, H, w.dtype if w_pre is not None else cast, x.device) if w_pre is not None or cast is not None else None
    assert (a is None or a.dtype == w.dtype) and (y2 is None or (y is not None and y2.dtype == y.dtype))
    check(_lib.lib().tfb_res_norm(ptr(ids), ptr(table), table.stride(0) if table is not None else 0, float(scale),
                                  table.shape[0] if table is not None else 0, x.data_ptr(), x.stride(0), ptr(y),
                                  y.stride(0) if y is not None else 0, ptr(y2), y2.stride(0) if y2 is not None else 0, ptr(w_post), ptr(b_post), ptr(scale_post), ptr(w_pre), ptr(b_pre), ptr(a),
                                  a.stride(0) if a is not None else 0, ptr(row_index), n, H, float(eps), NORM[kind], _f32(w), stream()),
          "res_norm")
    return a


def group_rms(x, w, groups, eps):
    """RMS norm of every one of ``groups`` equal consecutive parts of a row; the weight is the factor itself."""
    xf = x.float().unflatten(-1, (groups, -1))
    return (xf / torch.sqrt(xf.pow(2).mean(-1, keepdim=True) + eps)).flatten(-2) * w.float()


def stream_norm(x, eps, *, y=None, y2=None, w_post=None, w_post2=None, share=1.0, mix=None, out=None, w_in=None, w_pre=None, groups=1, ids=None,
                table=None, scale=1.0, row_index=None):
    """What stands between two sublayers over a residual of several streams, fp32 ``x`` [n, S, H], in place:
    x_t <- sum_s mix[s, t] x_s + out[t] y', with y' = share * (y + y2), each an RMS norm of itself first where it has a weight (``w_post``,
    ``w_post2``).  Returns group_rms(sum_s w_in[s] x_s; w_pre) in the weight's dtype (``w_in`` None: the plain sum), None without
    ``w_pre``.  ``ids``: all streams start as scale * table[ids].  ``row_index`` (int32): only those rows are computed and returned, and x
    keeps its values."""
    n, S, H = x.shape
    if not x.is_cuda:
        v = (table[ids.long()].float() * scale)[:, None].expand(-1, S, -1) if ids is not None else x
        if y is not None:
            z = (plain_rms(y, w_post, eps) if w_post is not None else y.float())
            if y2 is not None:
                z = z + (plain_rms(y2, w_post2, eps) if w_post2 is not None else y2.float())
            v = torch.einsum("nsh,st->nth", v, mix.float()) + out.float()[:, None] * (z * share)[:, None]
        if row_index is None:
            x.copy_(v)
        else:
            v = v[row_index.long()]
        if w_pre is None:
            return None
        u = v.sum(1) if w_in is None else torch.einsum("nsh,s->nh", v, w_in.float())
        return group_rms(u, w_pre, groups, eps).to(w_pre.dtype)
    n = n if row_index is None else row_index.shape[0]
    dt = next(t for t in (w_pre, table, y) if t is not None).dtype
    assert x.is_contiguous() and x.dtype == torch.float32 and dt in (torch.float32, torch.bfloat16)
    for t in (y, y2, w_post, w_post2, mix, out, w_in, w_pre, table):
        assert t is None or (t.dtype == dt and t.stride(-1) == 1)
    a = rows(n, H, dt, x.device) if w_pre is not None else None
    ld = lambda t: t.stride(0) if t is not None else 0
    check(_lib.lib().tfb_stream_norm(ptr(ids), ptr(table), ld(table), float(scale), table.shape[0] if table is not None else 0, x.data_ptr(), S, ptr(y),
                                     ld(y), ptr(y2), ld(y2), ptr(w_post), ptr(w_post2), float(share), ptr(mix), ptr(out), ptr(w_in), ptr(w_pre), groups,
                                     ptr(a), ld(a), ptr(row_index), n, H, float(eps), int(dt == torch.float32), stream()), "stream_norm")
    return a


def glu_silu(gu):
    return glu(gu, "silu")


def glu_ref(gu, act, limit=0.0):
    Fh = gu.shape[1] // 2
    g, u = gu[:, :Fh].float(), gu[:, Fh:].float()
    if act == "clamped":
        g = g.clamp(max=limit)
        return (g * torch.sigmoid(1.702 * g) * (u.clamp(-limit, limit) + 1)).to(gu.dtype)
    return ((g * torch.sigmoid(g) if act == "silu" else torch.nn.functional.gelu(g, approximate="tanh")) * u).to(gu.dtype)


def glu(gu, act, limit=0.0):
    """[gate | up] -> act(gate) * up; ``act``: "silu", "gelu_tanh" or "clamped": with g = min(gate, limit) and u = up clamped to
    +-limit, g sigmoid(1.702 g) (u + 1)."""
    M, F2 = gu.shape
    Fh = F2 // 2
    if not gu.is_cuda:
        return glu_ref(gu, act, limit)
    out = rows(M, Fh, gu.dtype, gu.device)
    check(_lib.lib().tfb_glu(gu.data_ptr(), gu.stride(0), out.data_ptr(), out.stride(0), M, Fh, GLU[act], float(limit), _f32(gu), stream()), "glu")
    return out


# ---------------------------------------------------------------------------------------------------- rotation + cache
def rope_append(qkv, tables, positions, nq, nk, D, dims, v_cols, slots=None, kpool=None, vpool=None, norms=None,
                q_factor=None):
    """Rotate the first ``dims`` entries of the nq query and nk key heads of every row of ``qkv`` ([q | k | v | ...]) in place and
    write k and v to flat slots of the pools ([slots, nk * D], [slots, v_cols]; negative slots are not cached).  ``norms``
    (weights of the queries, of the keys, eps; no weights: None, None, eps): every head is divided by its root mean square and weighted
    first; ``q_factor`` [nq] (with ``norms`` only) multiplies the normed query heads.  ``dims`` 0: no rotation (``tables`` None)."""
    assert q_factor is None or norms
    cos, sin = tables or (None, None)
    T = qkv.shape[0]
    if not qkv.is_cuda:
        half = dims // 2
        x = qkv[:, :(nq + nk) * D].reshape(T, nq + nk, D).float()
        if norms:
            one = torch.ones(D)
            q, k = (plain_rms(t, one if w is None else w, norms[2]) for t, w in ((x[:, :nq], norms[0]), (x[:, nq:], norms[1])))
            x = torch.cat([q if q_factor is None else q * q_factor.float()[:, None], k], 1)
        if dims:
            c, s = cos[positions.long()][:, None], sin[positions.long()][:, None]
            u, v = x[..., :half], x[..., half:dims]
            x = torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)
        if norms or dims:
            qkv[:, :(nq + nk) * D] = x.reshape(T, -1).to(qkv.dtype)
        if nk and slots is not None:
            keep = slots >= 0
            kpool[slots[keep]] = qkv[keep, nq * D:(nq + nk) * D]
            vpool[slots[keep]] = qkv[keep, (nq + nk) * D:(nq + nk) * D + v_cols]
        return qkv
    if norms:
        check(_lib.lib().tfb_norm_rope_append(qkv.data_ptr(), qkv.stride(0), ptr(norms[0]), ptr(norms[1]), ptr(q_factor), float(norms[2]), ptr(cos),
                                              ptr(sin), cos.shape[0] if dims else 0, positions.data_ptr(), ptr(slots), ptr(kpool), ptr(vpool),
                                              kpool.shape[0] if kpool is not None else 0, T, nq, nk, D, dims, v_cols, _f32(qkv), stream()),
              "norm_rope_append")
        return qkv
    check(_lib.lib().tfb_rope_append(qkv.data_ptr(), qkv.stride(0), ptr(cos), ptr(sin), cos.shape[0] if dims else 0, positions.data_ptr(),
                                     ptr(slots), ptr(kpool), ptr(vpool), kpool.shape[0] if kpool is not None else 0, T, nq, nk, D, dims,
                                     v_cols, _f32(qkv), stream()), "rope_append")
    return qkv


def gather_rows(pool, pages, lo, n):
    """Cached rows of positions lo .. lo + n - 1 of one sequence (``pages``: its page list, int32), contiguous."""
    width = pool.shape[1]
    if not pool.is_cuda:
        p = torch.arange(lo, lo + n)
        return pool[pages[p // PAGE].long() * PAGE + p % PAGE].clone()
    out = torch.empty((n, width), dtype=pool.dtype, device=pool.device)
    check(_lib.lib().tfb_gather_rows(pool.data_ptr(), pool.shape[0], pages.data_ptr(), PAGE, lo, n, out.data_ptr(), width, _f32(pool), stream()),
          "gather_rows")
    return out


# ---------------------------------------------------------------------------------------------------- differential attention
def _diff_ref(q, k, v, B, S, Skv, H, G, D, V, window, scale, lam, out_scale, eps):
    R = H // G
    Q = q.reshape(B, S, H, 2, D).permute(0, 2, 3, 1, 4).float()                     # [B, H, 2, S, D]
    K = k.reshape(B, Skv, G, 2, D).permute(0, 2, 3, 1, 4).float().repeat_interleave(R, 1)
    W = v.reshape(B, Skv, G, V).permute(0, 2, 1, 3).float().repeat_interleave(R, 1)
    i = torch.arange(S)[:, None] + (Skv - S)
    j = torch.arange(Skv)[None]
    hide = (j > i) | ((i - j >= window) if window else torch.zeros(1, dtype=torch.bool))
    s = (Q @ K.transpose(-1, -2) * scale).masked_fill(hide, -math.inf)
    a = torch.softmax(s, -1) @ W[:, :, None]                                        # [B, H, 2, S, V]
    o = a[:, :, 0] - lam * a[:, :, 1]
    o = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps) * out_scale
    return o.permute(0, 2, 1, 3).reshape(B * S, H * V).to(q.dtype)


def diff_attn(q, k, v, B, S, Skv, H, G, D, V, window, scale, lam, out_scale, eps):
    """Differential attention of B prompts.  q [B*S, 2 H D], k [B*Skv, 2 G D] (rotated), v [B*Skv, G V]; the queries are the
    last S of the Skv positions; ``window`` 0: plain causal.  Returns [B*S, H V]."""
    if not q.is_cuda:
        return _diff_ref(q, k, v, B, S, Skv, H, G, D, V, window, scale, lam, out_scale, eps)
    o = rows(B * S, H * V, q.dtype, q.device)
    check(_lib.lib().tfb_diff_attn_fwd(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), o.data_ptr(), o.stride(0),
                                       B, S, Skv, H, G, D, V, window, float(scale), float(lam), float(out_scale), float(eps), _f32(q),
                                       _lib.status_word(q.device).data_ptr(), stream()), "diff_attn_fwd")
    return o


def diff_decode(q, kpool, vpool, block_table, positions, H, G, D, V, window, scale, lam, out_scale, eps, max_keys: int = 0,
                splits: Optional[int] = None):
    """One query per sequence (q [B, 2 H D], rotated, at ``positions``) over its cached rows.  ``max_keys``: a bound on the
    keys any query can see (for the choice of the split count only)."""
    B = q.shape[0]
    if not q.is_cuda:
        out = torch.zeros((B, H * V), dtype=q.dtype)
        for b in range(B):
            n = int(positions[b]) + 1
            lo = max(0, n - window) if window else 0
            p = torch.arange(lo, n)
            s = block_table[b, (p // PAGE).long()].long() * PAGE + p % PAGE
            out[b] = _diff_ref(q[b:b + 1], kpool[s], vpool[s], 1, 1, n - lo, H, G, D, V, window, scale, lam, out_scale, eps)[0]
        return out
    o = rows(B, H * V, q.dtype, q.device)
    L, f32 = _lib.lib(), _f32(q)
    acc = ml = None
    if L.tfb_diff_decode_tc(D, V, f32) and q.stride(0) % 8 == 0:
        chunks = (H // G + 7) // 8
        if splits is None:
            keys = max_keys or block_table.shape[1] * PAGE
            keys = min(keys, window + PAGE) if window else keys
            splits = max(1, min(32, (4 * 148) // max(1, B * G * chunks), keys // 128))
        acc = torch.empty(B * G * chunks * splits * 16 * V, dtype=torch.float32, device=q.device)
        ml = torch.empty(B * G * chunks * splits * 32, dtype=torch.float32, device=q.device)
    check(L.tfb_diff_decode(q.data_ptr(), q.stride(0), kpool.data_ptr(), vpool.data_ptr(), kpool.shape[0], block_table.data_ptr(),
                            block_table.shape[1], PAGE, positions.data_ptr(), o.data_ptr(), o.stride(0), ptr(acc), ptr(ml), splits or 1, B, H, G,
                            D, V, window, float(scale), float(lam), float(out_scale), float(eps), f32, _lib.status_word(q.device).data_ptr(),
                            stream()), "diff_decode", 2 if acc is not None else 1)
    return o


# ---------------------------------------------------------------------------------------------------- softmax attention with options
class HeadOptions(NamedTuple):
    """``window`` > 0: a query sees that many keys up to its own, and the first ``keep_first`` of the sequence; ``softcap`` > 0: scores
    become cap tanh(score / cap); ``sink``: one more key of score 0 in the denominator; the query at position p is multiplied by
    1 + temp_coef ln(floor((p + 1) / temp_every) + 1); ``chunk`` > 0 (no window then): it sees the keys of its own chunk of so many
    positions, counted from 0, and those first ones."""
    window: int = 0
    keep_first: int = 0
    softcap: float = 0.0
    sink: bool = False
    temp_coef: float = 0.0
    temp_every: int = 1
    chunk: int = 0

    def first_key(self, i: int) -> int:
        """The first key that the query at position i sees, kept ones aside."""
        return max(0, i - self.window + 1) if self.window else i // self.chunk * self.chunk if self.chunk else 0

    def args(self, sinks):
        """Of the entry points: window, chunk, keep, cap, sink, sinks, temp."""
        return self.window, self.chunk, self.keep_first, self.softcap, 2 if sinks is not None else int(self.sink), ptr(sinks), self.temp_coef, self.temp_every


PLAIN = HeadOptions()


def _head_attn_ref(q, k, v, B, S, Skv, H, G, D, V, scale, gate=None, opt=PLAIN, pos0=0, sinks=None):
    R = H // G
    Q = q.reshape(B, S, H, D).transpose(1, 2).float()
    K = k.reshape(B, Skv, G, D).transpose(1, 2).float().repeat_interleave(R, 1)
    W = v.reshape(B, Skv, G, V).transpose(1, 2).float().repeat_interleave(R, 1)
    i, j = torch.arange(S)[:, None] + (Skv - S), torch.arange(Skv)[None]
    hide = j > i
    if opt.window:
        hide = hide | ((i - j >= opt.window) & (j >= opt.keep_first))
    if opt.chunk:
        hide = hide | ((i // opt.chunk != j // opt.chunk) & (j >= opt.keep_first))
    temp = 1 + opt.temp_coef * torch.log(((torch.arange(S) + pos0 + 1) // opt.temp_every + 1).float())
    s = Q * temp[:, None] @ K.transpose(-1, -2) * scale
    if opt.softcap:
        s = opt.softcap * torch.tanh(s / opt.softcap)
    s = s.masked_fill(hide, -math.inf)
    if opt.sink or sinks is not None:
        s = torch.cat([s, torch.zeros(B, H, S, 1) if sinks is None else sinks.float()[:, None, None].expand(B, H, S, 1)], -1)
        W = torch.cat([W, torch.zeros(B, H, 1, V)], 2)
    o = (torch.softmax(s, -1) @ W).transpose(1, 2)                                 # [B, S, H, V]
    if gate is not None:
        o = o * torch.sigmoid(gate.float()).reshape(B, S, H, -1)
    return o.reshape(B * S, H * V).to(q.dtype)


def head_attn(q, k, v, B, S, Skv, H, G, D, V, scale, gate=None, opt=PLAIN, pos0=0, sinks=None):
    """Causal softmax attention of B prompts whose keys and values may have different sizes.  q [B*S, H D], k [B*Skv, G D],
    v [B*Skv, G V]; the queries are the last S of the Skv keys and stand at positions pos0 ... (with a window, keys between the
    kept ones and the window of the first query may be left out; with chunks and no kept ones those of earlier chunks);
    ``gate`` [B*S, H] or [B*S, H V]: heads, or their entries, are multiplied by its sigmoid; ``sinks`` [H]: the score of one more key per
    head in the denominator.  Returns [B*S, H V]."""
    if not q.is_cuda:
        return _head_attn_ref(q, k, v, B, S, Skv, H, G, D, V, scale, gate, opt, pos0, sinks)
    assert sinks is None or sinks.dtype == q.dtype
    o = rows(B * S, H * V, q.dtype, q.device)
    check(_lib.lib().tfb_head_attn(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), o.data_ptr(), o.stride(0),
                                   ptr(gate), gate.stride(0) if gate is not None else 0, int(gate is not None and gate.shape[1] != H), B, S, Skv, H,
                                   G, D, V, float(scale), *opt.args(sinks), pos0,
                                   _f32(q), _lib.status_word(q.device).data_ptr(), stream()), "head_attn")
    return o


def head_decode(q, kpool, vpool, block_table, positions, H, G, D, V, scale, gate=None, opt=PLAIN, splits: Optional[int] = None,
                sinks=None):
    """One query per sequence (q [B, H D] at ``positions``) over its cached rows (pools [slots, G D] and [slots, G V]); ``gate`` [B, H]
    or [B, H V]; ``sinks`` [H]."""
    B = q.shape[0]
    if not q.is_cuda:
        out = torch.zeros((B, H * V), dtype=q.dtype)
        for b in range(B):
            n = int(positions[b]) + 1
            lo = opt.first_key(n - 1)
            p = torch.cat([torch.arange(min(opt.keep_first, lo)), torch.arange(lo, n)])
            s = block_table[b, (p // PAGE).long()].long() * PAGE + p % PAGE
            out[b] = _head_attn_ref(q[b:b + 1], kpool[s], vpool[s], 1, 1, len(p), H, G, D, V, scale, gate[b:b + 1] if gate is not None else None,
                                    opt._replace(window=0, chunk=0), n - 1, sinks)[0]
        return out
    assert sinks is None or sinks.dtype == q.dtype
    L, f32 = _lib.lib(), _f32(q)
    o = rows(B, H * V, q.dtype, q.device)
    acc = ml = None
    keys = block_table.shape[1] * PAGE
    keys = min(keys, (opt.window or opt.chunk) + opt.keep_first) if opt.window or opt.chunk else keys
    n = L.tfb_head_decode_plan(B, H, G, D, V, keys, f32)         # key splits of the tensor-core form, 0: the other form
    if n and q.stride(0) % 8 == 0:
        splits = splits or n
        acc = torch.empty(B * H * splits * V, dtype=torch.float32, device=q.device)
        ml = torch.empty(B * H * splits * 2, dtype=torch.float32, device=q.device)
    check(L.tfb_head_decode(q.data_ptr(), q.stride(0), kpool.data_ptr(), vpool.data_ptr(), kpool.shape[0], block_table.data_ptr(),
                            block_table.shape[1], PAGE, positions.data_ptr(), o.data_ptr(), o.stride(0), ptr(gate),
                            gate.stride(0) if gate is not None else 0, int(gate is not None and gate.shape[1] != H), ptr(acc), ptr(ml), splits or 1, B,
                            H, G, D, V, float(scale), *opt.args(sinks), f32,
                            _lib.status_word(q.device).data_ptr(), stream()), "head_decode", 2 if acc is not None else 1)
    return o


# ---------------------------------------------------------------------------------------------------- latent attention
def latent_append(c, w, eps, slots, pool, want_rows=True):
    """Rows c [T, R] divided by their root mean square and weighted with w, written to flat slots of ``pool`` [slots, R padded to 8]
    (negative slots are not cached; ``slots`` None: nothing is).  Returns the rows, or None without ``want_rows``."""
    T, R = c.shape
    if not c.is_cuda:
        cf = c.float()
        v = (cf / torch.sqrt(cf.pow(2).mean(-1, keepdim=True) + eps) * w.float()).to(c.dtype)
        if slots is not None:
            keep = slots >= 0
            pool[slots[keep], :R] = v[keep]
        return v
    out = rows(T, R, c.dtype, c.device) if want_rows else None
    check(_lib.lib().tfb_latent_append(c.data_ptr(), c.stride(0), w.data_ptr(), float(eps), ptr(slots), ptr(out), out.stride(0) if want_rows else 0,
                                       pool.data_ptr(), pool.shape[0], pool.shape[1], T, R, _f32(c), stream()), "latent_append")
    return out


def head_linear(x, w, heads, k, n, gate=None, transposed=False):
    """One small product per head: x [M, heads * k] with w of heads blocks [n, k] ([k, n] when ``transposed``) stacked on the rows
    -> [M, heads * n8] where n8 is n for plain and n rounded up to 8 (zero filled) for transposed blocks; ``gate`` [M, heads]: head h
    is multiplied by sigmoid(gate[:, h]) (plain blocks only).  Plain blocks: x comes with every head padded to a multiple of 8 entries
    with zeros (as ``latent_decode`` returns it)."""
    M = x.shape[0]
    n8 = (n + 7) // 8 * 8 if transposed else n
    if not x.is_cuda:
        W = w.float().reshape(heads, k, n).transpose(1, 2) if transposed else w.float().reshape(heads, n, k)
        k_in = x.shape[1] // heads                       # rows of an earlier product may be padded
        o = torch.einsum("mhk,hnk->mhn", x.float().reshape(M, heads, k_in)[..., :k], W)
        if gate is not None:
            o = o * torch.sigmoid(gate.float())[..., None]
        out = torch.zeros((M, heads, n8), dtype=x.dtype)
        out[..., :n] = o.to(x.dtype)
        return out.view(M, heads * n8)
    L, x_head = _lib.lib(), x.shape[1] // heads
    assert gate is None or not transposed
    if x.dtype == torch.float32:
        out = torch.zeros((M, heads * n8), dtype=x.dtype, device=x.device)
        check(L.tfb_gemm_f32_heads(x.data_ptr(), x.stride(0), x_head, w.data_ptr(), w.stride(0), int(transposed), out.data_ptr(), out.stride(0), n8,
                                   ptr(gate), gate.stride(0) if gate is not None else 0, M, heads, n, k, stream()), "gemm_f32_heads")
        return out
    out = rows(M, heads * n8, x.dtype, x.device)
    if transposed:
        check(L.tfb_head_linear(x.data_ptr(), x.stride(0), x_head, w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0), n8, M, heads, n, k,
                                stream()), "head_linear")
    else:                                      # k rounded up to 8: the padding of x is zero and that of w finite
        k8 = (k + 7) // 8 * 8
        assert x_head >= k8 and w.stride(0) >= k8
        check(L.tfb_skinny_linear_heads(x.data_ptr(), x.stride(0), x_head, w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0), ptr(gate),
                                        gate.stride(0) if gate is not None else 0, M, heads, n, k8, 0, stream()), "skinny_linear_heads")
    return out


def latent_decode(q, pool, block_table, positions, H, R, scale, splits: Optional[int] = None):
    """One query per sequence and head over the cached latents, which are keys and values of every head at once: q [B, H * R8] (in the
    latent space, R8 = R padded to 8 with zeros, at ``positions``), pool [slots, R8].  Returns softmax(scale q c) c, [B, H * R8]."""
    B, W = q.shape[0], pool.shape[1]
    if not q.is_cuda:
        out = torch.zeros((B, H, W), dtype=q.dtype)
        for b in range(B):
            p = torch.arange(int(positions[b]) + 1)
            c = pool[block_table[b, (p // PAGE).long()].long() * PAGE + p % PAGE].float()
            out[b] = (torch.softmax(q[b].float().view(H, W) @ c.t() * scale, -1) @ c).to(q.dtype)
        return out.view(B, H * W)
    L, f32 = _lib.lib(), _f32(q)
    o = rows(B, H * W, q.dtype, q.device)
    acc = ml = None
    s = L.tfb_latent_decode_plan(B, H, W, block_table.shape[1] * PAGE, f32)      # key splits of the tensor-core form, 0: the other form
    if s:
        s = splits or s
        acc = torch.empty(B * H * s * W if s > 1 else 0, dtype=torch.float32, device=q.device)
        ml = torch.empty(B * H * s * 2 if s > 1 else 0, dtype=torch.float32, device=q.device)
    check(L.tfb_latent_decode(q.data_ptr(), q.stride(0), pool.data_ptr(), pool.shape[0], block_table.data_ptr(), block_table.shape[1], PAGE,
                              positions.data_ptr(), o.data_ptr(), o.stride(0), ptr(acc), ptr(ml), s, B, H, R, W, float(scale), f32,
                              _lib.status_word(q.device).data_ptr(), stream()), "latent_decode", 1 + int(s > 1))
    return o


# ---------------------------------------------------------------------------------------------------- gated delta rule
@dataclass
class DeltaRows:
    """Prepared rows of B sequences: on CUDA the kernels' own layouts (see csrc/kernels/delta_rule.cu), ``pair`` holding k.q
    when every sequence has one row; on the CPU q, k [T, G, D], v [T, H, V], decay, beta [T, H]."""
    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor
    decay: torch.Tensor
    beta: torch.Tensor
    pair: Optional[torch.Tensor] = None
    coef: Optional[torch.Tensor] = None


def _step_fits(D, V) -> bool:
    return V % 4 == 0 and V <= 256 and D <= 256 and (V <= 128 or D <= 128)


def delta_prep(proj, conv_w, conv_state, state_slots, A_log, dt_bias, lens, B, S, G, H, D, V, has_past, step=False) -> DeltaRows:
    """proj [B*S, 2 G D + 2 H V + 2 H] = q | k | v | gate | b | a  ->  convolved, activated, unit-length rows and gates, all
    fp32.  ``conv_state`` [slots, taps - 1, channels] is read for sequences that go on (``has_past``) and left holding their last
    inputs.  ``step``: the rows are for ``delta_step`` (one token per sequence)."""
    T, C, taps = B * S, 2 * G * D + H * V, conv_w.shape[1]
    if not proj.is_cuda:
        x = proj[:, :C].reshape(B, S, C)
        n = lens if lens is not None else torch.full((B,), S)
        full = torch.zeros((B, taps - 1 + S, C), dtype=x.dtype)
        full[:, taps - 1:] = x
        if taps > 1 and has_past:
            ok = state_slots >= 0
            full[ok, :taps - 1] = conv_state[state_slots[ok].long()]
        w = conv_w.float()
        y = sum(full[:, j:j + S].float() * w[:, j] for j in range(taps))
        y = (y * torch.sigmoid(y)).reshape(T, C)
        if taps > 1:
            for b in range(B):
                if int(state_slots[b]) >= 0:
                    conv_state[int(state_slots[b])] = full[b, int(n[b]): int(n[b]) + taps - 1]
        q, k = y[:, :G * D].reshape(T, G, D), y[:, G * D:2 * G * D].reshape(T, G, D)
        q = q / torch.sqrt(q.pow(2).sum(-1, keepdim=True) + 1e-6) * D ** -0.5
        k = k / torch.sqrt(k.pow(2).sum(-1, keepdim=True) + 1e-6)
        tail = proj[:, C + H * V:].float()
        beta = torch.sigmoid(tail[:, :H])
        decay = torch.exp(-torch.exp(A_log.float()) * torch.nn.functional.softplus(tail[:, H:2 * H] + dt_bias.float()))
        return DeltaRows(q, k, y[:, 2 * G * D:].reshape(T, H, V), decay, beta)
    L = _lib.lib()
    Dp, Vp = L.tfb_delta_padded_dim(D), (V + 3) // 4 * 4
    Sp = 1 if step and _step_fits(D, V) else (S + 3) // 4 * 4
    e = lambda *shape: torch.empty(shape, dtype=torch.float32, device=proj.device)
    r = DeltaRows(e(B, G, Sp, Dp), e(B, G, Sp, Dp), e(B, H, Sp, Vp), e(B, H, Sp), e(B, H, Sp))
    r.pair = e(B, G) if Sp == 1 else e(B, G, Sp // 4, 16)
    r.coef = None if Sp == 1 else e(B, H, Sp // 4, 32)
    check(L.tfb_delta_prep(proj.data_ptr(), proj.stride(0), conv_w.data_ptr(), ptr(conv_state), ptr(state_slots),
                           conv_state.shape[0] if conv_state is not None else 0, A_log.data_ptr(), dt_bias.data_ptr(), ptr(lens), r.q.data_ptr(),
                           r.k.data_ptr(), r.v.data_ptr(), r.decay.data_ptr(), r.beta.data_ptr(), r.pair.data_ptr(), ptr(r.coef), B, S, Sp, G, H,
                           D, V, taps, int(has_past), _f32(proj), stream()), "delta_prep", 1 + int(S > 1 and taps > 1) + int(Sp > 1))
    return r


def delta_scan(rows_: DeltaRows, state, state_slots, lens, B, S, G, H, D, V, has_past):
    """The recurrence over prepared rows; ``state`` [slots, H, D, V] fp32 is read (``has_past``) and updated.  Returns fp32
    [B*S, H, V] (rows past a sequence's length are zero)."""
    r = rows_
    if not r.q.is_cuda:
        out = torch.zeros(B * S, H, V)
        n = lens if lens is not None else torch.full((B,), S)
        rep = H // G
        for b in range(B):
            sl = int(state_slots[b])
            st = state[sl].clone() if has_past and sl >= 0 else torch.zeros(H, D, V)
            for t in range(b * S, b * S + int(n[b])):
                kk, qq = r.k[t].repeat_interleave(rep, 0), r.q[t].repeat_interleave(rep, 0)
                st = st * r.decay[t][:, None, None]
                u = r.beta[t][:, None] * (r.v[t] - torch.einsum("hdv,hd->hv", st, kk))
                st = st + kk[:, :, None] * u[:, None, :]
                out[t] = torch.einsum("hdv,hd->hv", st, qq)
            if sl >= 0:
                state[sl] = st
        return out
    o = torch.empty((B * S, H, V), dtype=torch.float32, device=r.q.device)
    check(_lib.lib().tfb_delta_scan(r.q.data_ptr(), r.k.data_ptr(), r.v.data_ptr(), r.coef.data_ptr(), o.data_ptr(), state.data_ptr(),
                                    state_slots.data_ptr(), state.shape[0], ptr(lens), B, S, G, H, D, V, int(has_past),
                                    _lib.status_word(o.device).data_ptr(), stream()), "delta_scan")
    return o


def gated_norm(o, gate, w, eps, dtype=None):
    """o [T, H, V] fp32 -> o / rms(o) [* w [V]] [* silu(gate [T, H V])], [T, H V] in ``dtype`` (that of the gate, if there is one)."""
    T, H, V = o.shape
    dtype = gate.dtype if gate is not None else dtype
    if not o.is_cuda:
        y = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps)
        if w is not None:
            y = y * w.float()
        if gate is not None:
            g = gate.reshape(T, H, V).float()
            y = y * (g * torch.sigmoid(g))
        return y.reshape(T, H * V).to(dtype)
    out = rows(T, H * V, dtype, o.device)
    assert w is None or w.dtype == dtype
    check(_lib.lib().tfb_gated_norm(o.data_ptr(), ptr(gate), gate.stride(0) if gate is not None else 0, ptr(w), out.data_ptr(), out.stride(0), T, H, V,
                                    float(eps), _f32(out), stream()), "gated_norm")
    return out


def delta_step(rows_: DeltaRows, state, state_slots, gate, w, eps, B, G, H, D, V, has_past=True):
    """One token per sequence (rows prepared with ``step``) with the gated norm of its output; [B, H V]."""
    r = rows_
    if not r.q.is_cuda or not _step_fits(D, V):
        return gated_norm(delta_scan(r, state, state_slots, None, B, 1, G, H, D, V, has_past), gate, w, eps)
    out = rows(B, H * V, gate.dtype, r.q.device)
    check(_lib.lib().tfb_delta_step(r.q.data_ptr(), r.k.data_ptr(), r.v.data_ptr(), r.pair.data_ptr(), r.decay.data_ptr(), r.beta.data_ptr(),
                                    state.data_ptr(), state_slots.data_ptr(), state.shape[0], gate.data_ptr(), gate.stride(0), w.data_ptr(),
                                    out.data_ptr(), out.stride(0), B, G, H, D, V, int(has_past), float(eps), _f32(gate), stream()), "delta_step")
    return out


# ---------------------------------------------------------------------------------------------------- linear attention with decays
@dataclass
class GlaRows:
    """Prepared rows of B sequences.  On CUDA the scan's own layouts (see csrc/kernels/gated_linear.cu): per four tokens queries times
    the decays up to them, keys times those behind them, the decay over all four, and the products between them; on the CPU q, k,
    decay [T, H, D], v [T, H, V]."""
    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor
    decay: torch.Tensor
    pair: Optional[torch.Tensor] = None


def _gla_rows(B, S, H, D, V, device):
    Dp, Vp, n4 = next((d for d in (32, 64, 128, 256, 512) if D <= d), 0), (V + 3) // 4 * 4, (S + 3) // 4
    e = lambda *shape: torch.empty(shape, dtype=torch.float32, device=device)
    return GlaRows(e(B, H, 4 * n4, Dp), e(B, H, 4 * n4, Dp), e(B, H, 4 * n4, Vp), e(B, H, n4, Dp), e(B, H, n4, 16)), Dp


def _ptrs(r: GlaRows):
    return r.q.data_ptr(), r.k.data_ptr(), r.v.data_ptr(), r.decay.data_ptr(), r.pair.data_ptr()


def gla_prep(proj, a2, bias, tau, lens, B, S, H, D, V) -> GlaRows:
    """proj [B*S, 2 H D + 2 H V + rank] = q | k | v | gate | a1, a2 [H D, rank], bias [H D]: scaled queries, decays
    sigmoid(a2 a1 + bias)^(1/tau) and rows for ``gla_scan``, all fp32."""
    if not proj.is_cuda:
        T, n = proj.shape[0], H * D
        x = proj.float()
        z = x[:, 2 * n + 2 * H * V:] @ a2.float().t() + bias.float()
        return GlaRows(x[:, :n].reshape(T, H, D) * D ** -0.5, x[:, n:2 * n].reshape(T, H, D), x[:, 2 * n:2 * n + H * V].reshape(T, H, V),
                       torch.exp(torch.nn.functional.logsigmoid(z) / tau).reshape(T, H, D))
    r, Dp = _gla_rows(B, S, H, D, V, proj.device)
    check(_lib.lib().tfb_gla_prep(proj.data_ptr(), proj.stride(0), a2.data_ptr(), a2.stride(0), bias.data_ptr(), a2.shape[1], float(tau), ptr(lens),
                                  *_ptrs(r), B, S, H, D, Dp, V, _f32(proj), stream()), "gla_prep")
    return r


def forget_prep(proj, bias, lower, lens, B, S, H, D, V) -> GlaRows:
    """proj [B*S, 2 H D + H V ...] = q | f | v ..., bias, lower [H D]: queries silu(q), decays a = lower + (1 - lower) sigmoid(f + bias), keys
    1 - a; rows for ``gla_scan``, all fp32."""
    if not proj.is_cuda:
        T, n = proj.shape[0], H * D
        x, l = proj.float(), lower.float()
        z = x[:, n:2 * n] + bias.float()
        return GlaRows((x[:, :n] * torch.sigmoid(x[:, :n])).reshape(T, H, D), ((1 - l) * torch.sigmoid(-z)).reshape(T, H, D),
                       x[:, 2 * n:2 * n + H * V].reshape(T, H, V), (l + (1 - l) * torch.sigmoid(z)).reshape(T, H, D))
    r, Dp = _gla_rows(B, S, H, D, V, proj.device)
    check(_lib.lib().tfb_forget_prep(proj.data_ptr(), proj.stride(0), bias.data_ptr(), lower.data_ptr(), ptr(lens), *_ptrs(r), B, S, H, D, Dp, V,
                                     _f32(proj), stream()), "forget_prep")
    return r


def retention_prep(proj, decay, tables, dims, positions, lens, B, S, H, D, V) -> GlaRows:
    """proj [B*S, 2 H D + H V ...] = q | k | v ..., decay [H] fp32: q and k rotated by their positions (first ``dims`` entries, 0: no
    rotation), k scaled by D^(-1/2); rows for ``gla_scan``, all fp32."""
    cos, sin = tables or (None, None)
    if not proj.is_cuda:
        T, n, half = proj.shape[0], H * D, dims // 2
        x = proj.float()
        qk = x[:, :2 * n].reshape(T, 2 * H, D)
        if dims:
            c, s = cos[positions.long()][:, None], sin[positions.long()][:, None]
            u, v = qk[..., :half], qk[..., half:dims]
            qk = torch.cat([u * c - v * s, v * c + u * s, qk[..., dims:]], -1)
        return GlaRows(qk[:, :H], qk[:, H:] * D ** -0.5, x[:, 2 * n:2 * n + H * V].reshape(T, H, V), decay[:, None].expand(T, H, D))
    r, Dp = _gla_rows(B, S, H, D, V, proj.device)
    check(_lib.lib().tfb_retention_prep(proj.data_ptr(), proj.stride(0), decay.data_ptr(), ptr(cos), ptr(sin), cos.shape[0] if dims else 0, dims,
                                        positions.data_ptr(), ptr(lens), *_ptrs(r), B, S, H, D, Dp, V, _f32(proj), stream()), "retention_prep")
    return r


def gla_scan(rows_: GlaRows, state, state_slots, lens, B, S, H, D, V, has_past, segments: Optional[int] = None):
    """S <- diag(decay) S + k v^T, o = S^T q over prepared rows; ``state`` [slots, H, D, V] fp32 is read (``has_past``) and updated.
    Returns fp32 [B*S, H, V] (rows past a sequence's length are zero).  ``segments``: parts of a sequence that run side by side (None: the
    kernel's choice)."""
    r = rows_
    if not r.q.is_cuda:
        out = torch.zeros(B * S, H, V)
        n = lens if lens is not None else torch.full((B,), S)
        for b in range(B):
            sl = int(state_slots[b])
            st = state[sl].clone() if has_past and sl >= 0 else torch.zeros(H, D, V)
            for t in range(b * S, b * S + int(n[b])):
                st = st * r.decay[t][..., None] + r.k[t][..., None] * r.v[t][:, None]
                out[t] = torch.einsum("hdv,hd->hv", st, r.q[t])
            if sl >= 0:
                state[sl] = st
        return out
    o = torch.empty((B * S, H, V), dtype=torch.float32, device=r.q.device)
    L = _lib.lib()
    n = segments or L.tfb_gla_scan_segments(B, S, H, D, V)
    work = torch.empty(B * n * H * (D * V + r.q.shape[-1]), dtype=torch.float32, device=o.device) if n > 1 else None
    check(L.tfb_gla_scan(*_ptrs(r), o.data_ptr(), state.data_ptr(), state.shape[0], state_slots.data_ptr(), B, S, H, D, V, int(has_past), ptr(lens), n,
                         ptr(work), _lib.status_word(o.device).data_ptr(), stream()), "gla_scan", 1 + int(n > 1))
    return o


def _gate(proj, H, D, V):
    return proj[:, 2 * H * D + H * V:2 * H * D + 2 * H * V]


def gla_step(proj, a2, bias, tau, state, state_slots, w, eps, B, H, D, V):
    """One token per sequence: decays, recurrence and the gated norm of its output; [B, H V]."""
    gate = _gate(proj, H, D, V)
    if not proj.is_cuda or not _step_fits(D, V):
        return gated_norm(gla_scan(gla_prep(proj, a2, bias, tau, None, B, 1, H, D, V), state, state_slots, None, B, 1, H, D, V, True), gate, w, eps)
    out = rows(B, H * V, proj.dtype, proj.device)
    check(_lib.lib().tfb_gla_step(proj.data_ptr(), proj.stride(0), a2.data_ptr(), a2.stride(0), bias.data_ptr(), a2.shape[1], float(tau),
                                  state.data_ptr(), state_slots.data_ptr(), state.shape[0], w.data_ptr(), out.data_ptr(), out.stride(0), B, H, D, V,
                                  float(eps), _f32(proj), stream()), "gla_step")
    return out


def forget_step(proj, bias, lower, state, state_slots, w, eps, B, H, D, V, gated=False):
    """One token per sequence, as ``gla_step``; [B, H V].  ``gated``: v is followed by the gate."""
    if not proj.is_cuda or not _step_fits(D, V):
        o = gla_scan(forget_prep(proj, bias, lower, None, B, 1, H, D, V), state, state_slots, None, B, 1, H, D, V, True)
        return gated_norm(o, _gate(proj, H, D, V) if gated else None, w, eps, proj.dtype)
    out = rows(B, H * V, proj.dtype, proj.device)
    check(_lib.lib().tfb_forget_step(proj.data_ptr(), proj.stride(0), bias.data_ptr(), lower.data_ptr(), int(gated), state.data_ptr(),
                                     state_slots.data_ptr(), state.shape[0], ptr(w), out.data_ptr(), out.stride(0), B, H, D, V, float(eps), _f32(proj),
                                     stream()), "forget_step")
    return out


def retention_step(proj, decay, tables, dims, positions, state, state_slots, w, eps, B, H, D, V, gated=True):
    """One token per sequence, as ``gla_step``; [B, H V]."""
    cos, sin = tables or (None, None)
    if not proj.is_cuda or not _step_fits(D, V):
        o = gla_scan(retention_prep(proj, decay, tables, dims, positions, None, B, 1, H, D, V), state, state_slots, None, B, 1, H, D, V, True)
        return gated_norm(o, _gate(proj, H, D, V) if gated else None, w, eps, proj.dtype)
    out = rows(B, H * V, proj.dtype, proj.device)
    check(_lib.lib().tfb_retention_step(proj.data_ptr(), proj.stride(0), decay.data_ptr(), ptr(cos), ptr(sin), cos.shape[0] if dims else 0, dims,
                                        positions.data_ptr(), int(gated), state.data_ptr(), state_slots.data_ptr(), state.shape[0], ptr(w),
                                        out.data_ptr(), out.stride(0), B, H, D, V, float(eps), _f32(proj), stream()), "retention_step")
    return out
