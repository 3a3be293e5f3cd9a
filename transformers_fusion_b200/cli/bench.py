"""quant_bench: ``--kernel <name> --size N`` times one device kernel; ``--inference --model m.quant --prompt p``
times generation (tools/bench.cpp:20-185).  Kernel timing: CUDA events on the launching stream, warm-up, an
L2-sized write between timed launches, best and median of ``--iters`` launches; rates are also printed as a
fraction of the copy / GEMM peaks when ``--peaks <json>`` (keys hbm_gbs, bf16_tflops) is given.

Kernels: gemm, gemm_nt_wgrad, gemm_fp8, attention_fwd, attention_bwd, rmsnorm, rmsnorm_bwd, swiglu, rope,
cross_entropy, adamw, paged_decode, sampling, moe_ffn; those of stack models (``STACK_KERNELS``): diff_attention,
diff_attention_window, attention_fwd_gqa128 (the plain form of the same layer), diff_decode, delta_prep, delta_scan,
delta_scan_one, gated_norm, delta_prep_step, delta_step, res_norm, glu_silu, rope_append; those of latent attention and the serving
mixture with the like kernels of the mixture-of-experts decoder (``LATENT_KERNELS``); those of attention with options and gated linear
attention (``GATED_KERNELS``); those of chunked attention, HGRN2, retention and streams of residuals (``STREAM_KERNELS``).  ``--kernel`` takes names and the
groups all, stack, latent, gated, streams, with commas between them.  ``--comm`` (multi-GPU) times the fused compute+collective kernels
against their NCCL forms (cli/bench_comm.py)."""
from __future__ import annotations

import argparse
import json
import statistics
import sys
import time

from .common import add_int

KERNELS = ("gemm", "gemm_wgrad", "gemm_fp8", "attention_fwd", "attention_bwd", "rmsnorm", "rmsnorm_bwd", "swiglu", "rope",
           "cross_entropy", "adamw", "paged_decode", "sampling", "moe_ffn")
STACK_KERNELS = ("diff_attention", "diff_attention_window", "attention_fwd_gqa128", "diff_decode", "delta_prep", "delta_scan", "delta_scan_one",
                 "gated_norm", "delta_prep_step", "delta_step", "res_norm", "glu_silu", "rope_append")
LATENT_KERNELS = ("head_attn", "attention_fwd_mha128", "latent_decode", "latent_decode_32", "latent_append", "latent_append_step", "head_linear_q",
                  "head_linear_v", "output_norm", "layernorm", "linear_relu2", "linear_relu2_step", "route", "route_step", "router_topk", "expert_rows",
                  "moe_permute", "expert_gate_up", "expert_gate_up_step", "expert_down", "expert_down_step", "expert_glu", "expert_glu_step",
                  "weighted_sum", "moe_combine", "mixture", "mixture_step", "moe_ffn_step", "kv_append")
GATED_KERNELS = ("head_attn_cap", "head_attn_window", "head_attn_gqa", "head_decode", "head_decode_cap", "head_decode_window", "gla_prep", "gla_scan",
                 "gla_scan_one", "gla_step", "norm_rope_append", "parallel_norm", "glu_gelu", "grouped_route", "grouped_route_step", "weighted_sum_gated")
STREAM_KERNELS = ("head_attn_chunk", "head_decode_chunk", "unit_norm_append", "forget_prep", "forget_scan", "forget_step", "retention_prep", "retention_scan",
                  "forget_scan_one", "retention_scan_one", "retention_step", "head_norm", "stream_norm", "stream_norm_pair", "glu_clamped", "route_all", "route_all_step", "expert_glu_clamped")
FP32_FMA_PER_SM = 128          # fp32 FMA lanes of an SM (the scans are reported against them)


def _build_stack(kernel, n, dev):
    """One launch (or one prepared operator call) of a stack model's kernel; layer sizes of a 2048-wide model: 16 heads, 4 kv heads,
    two maps of 64 and values of 128; delta rule with 16 heads of 128 x 128.  ``n``: tokens per sequence (prompts; about 16 k
    tokens in all) or cached tokens (decoding, 64 sequences)."""
    import torch

    from ..ops import functional as F
    from ..ops import stack as K
    bf = torch.bfloat16
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dtype=bf: torch.randn(*s, device=dev, generator=g).to(dtype)
    H, G, D, V = 16, 4, 64, 128
    B = 1 if kernel == "delta_scan_one" else max(1, (1 << 14) // n)
    T = B * n
    if kernel in ("diff_attention", "diff_attention_window", "attention_fwd_gqa128"):
        qkv = rnd(T, (2 * H + 2 * G) * D + G * V)
        if kernel == "attention_fwd_gqa128":
            return (lambda: F.attn_fwd(qkv, qkv, qkv, B, n, H, G, 128, k_col0=H * 128, v_col0=(H + G) * 128)), 4.0 * B * H * n * n / 2 * 128, 2 * T * 2 * H * 128
        W = 1024 if kernel == "diff_attention_window" else 0
        keys = sum(min(i + 1, W or n) for i in range(n))
        c = 2 * H * D
        q, k, v = qkv[:, :c], qkv[:, c:c + 2 * G * D], qkv[:, c + 2 * G * D:]
        return (lambda: K.diff_attn(q, k, v, B, n, n, H, G, D, V, W, 0.125, 0.4, 0.5, 1e-5)), 4.0 * B * H * keys * (D + V), T * (qkv.shape[1] + H * V) * 2
    if kernel == "diff_decode":
        B, pages = 64, 64 * (n // 16)
        kp, vp = rnd(pages * 16, G * 2 * D), rnd(pages * 16, G * V)
        bt = torch.randperm(pages, device=dev, generator=g).int().view(B, -1).contiguous()
        pos, q = torch.full((B,), n - 1, dtype=torch.int32, device=dev), rnd(B, 2 * H * D)
        return (lambda: K.diff_decode(q, kp, vp, bt, pos, H, G, D, V, 0, 0.125, 0.4, 0.5, 1e-5)), 4.0 * B * H * n * (D + V), B * n * G * (2 * D + V) * 2
    if kernel in ("res_norm", "glu_silu", "rope_append"):
        T, Hd = 1 << 14, 2048
        if kernel == "res_norm":
            x, y, w = rnd(T, Hd, dtype=torch.float32), rnd(T, Hd), rnd(Hd)
            return (lambda: K.res_norm(x, 1e-5, y=y, w_post=w, w_pre=w)), 0.0, T * Hd * 12
        if kernel == "glu_silu":
            gu = rnd(T, 2 * 5632)
            return (lambda: K.glu_silu(gu)), 0.0, T * 5632 * 6
        qkv, tab = rnd(T, (2 * H + 2 * G) * D + G * V), F.rope_tables(D, T, device=dev)
        pos, slots = torch.arange(T, device=dev, dtype=torch.int32), torch.arange(T, device=dev)
        kp, vp = rnd(T, 2 * G * D), rnd(T, G * V)
        return (lambda: K.rope_append(qkv, tab, pos, 2 * H, 2 * G, D, D, G * V, slots, kp, vp)), 0.0, T * ((2 * H + 2 * G) * D * 4 + 2 * G * D * 2 + G * V * 4)
    step = kernel in ("delta_prep_step", "delta_step")
    if step:
        B, n, T = 64, 1, 64
    G = H
    D = V = 128
    C = 2 * G * D + H * V
    p = K.rows(T, C + H * V + 2 * H, bf, dev)
    p.copy_(rnd(T, p.shape[1]))
    conv, A, dtb, w = rnd(C, 4), torch.full((H,), -1.5, device=dev).to(bf), torch.zeros(H, device=dev).to(bf), torch.ones(V, device=dev).to(bf)
    cs, st = torch.zeros(B, 3, C, dtype=bf, device=dev), torch.zeros(B, H, D, V, device=dev)
    sl = torch.arange(B, dtype=torch.int32, device=dev)
    prep = lambda: K.delta_prep(p, conv, cs, sl, A, dtb, None, B, n, G, H, D, V, step, step=step)
    if kernel in ("delta_prep", "delta_prep_step"):
        return prep, 0.0, T * C * (2 + 4) + (T * C * 2 * 6 if step else 0)
    r = prep()
    gate = p[:, C:C + H * V]
    if kernel == "delta_step":
        return (lambda: K.delta_step(r, st, sl, gate, w, 1e-5, B, G, H, D, V)), 0.0, B * H * D * V * 8
    if kernel == "gated_norm":
        o = K.delta_scan(r, st, sl, None, B, n, G, H, D, V, False)
        return (lambda: K.gated_norm(o, gate, w, 1e-5)), 0.0, T * H * V * 8
    if kernel in ("delta_scan", "delta_scan_one"):
        return (lambda: K.delta_scan(r, st, sl, None, B, n, G, H, D, V, False)), 6.0 * T * H * D * V, T * (2 * G * D + 2 * H * V) * 4
    raise SystemExit(f"Error: unknown kernel '{kernel}'")


def _build_latent(kernel, n, dev):
    """The same for the kernels of latent attention and of the serving mixture, beside the like ones of the mixture-of-experts
    decoder (attention_fwd_mha128, layernorm, router_topk, moe_permute, moe_combine, moe_ffn_step, kv_append): 2048 wide, 16 heads of
    128 over latents of 512, 64 experts of 704, six per token.  ``n``: tokens per sequence (prompts; 16 k tokens in all) or
    cached tokens (decoding); *_step: 64 rows."""
    import torch

    from ..ops import functional as F
    from ..ops import moe as M
    from ..ops import stack as K
    bf = torch.bfloat16
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dtype=bf, scale=1.0: (torch.randn(*s, device=dev, generator=g) * scale).to(dtype)
    Hd, H, D, R, E, k, Fh = 2048, 16, 128, 512, 64, 6, 704
    T = 64 if kernel.endswith("_step") or kernel.startswith("head_linear") else 1 << 14
    if kernel in ("head_attn", "attention_fwd_mha128"):
        B = max(1, T // n)
        q, kv, fl = rnd(B * n, H * D + H), rnd(B * n, 2 * H * D), 4.0 * B * H * n * n / 2 * D
        if kernel == "head_attn":
            return (lambda: K.head_attn(q[:, :H * D], kv[:, :H * D], kv[:, H * D:], B, n, n, H, H, D, D, D ** -0.5, q[:, H * D:])), fl, B * n * 4 * H * D * 2
        return (lambda: F.attn_fwd(q, kv, kv, B, n, H, H, D, q_col0=0, k_col0=0, v_col0=H * D)), fl, B * n * 4 * H * D * 2
    if kernel in ("latent_decode", "latent_decode_32"):
        B, H = 64, 32 if kernel.endswith("32") else 16
        pages = B * (n // 16)
        pool, q = rnd(pages * 16, R), rnd(B, H * R)
        bt = torch.randperm(pages, device=dev, generator=g).int().view(B, -1).contiguous()
        pos = torch.full((B,), n - 1, dtype=torch.int32, device=dev)
        return (lambda: K.latent_decode(q, pool, bt, pos, H, R, D ** -0.5)), 4.0 * B * H * n * R, B * n * R * 2
    if kernel.startswith("latent_append") or kernel == "kv_append":
        slots = torch.randperm(T, device=dev, generator=g)
        if kernel == "kv_append":
            from ..inference.kv_cache import PagedKVCache
            kv, qkv = PagedKVCache(1, T // 16, 4, 128, "bf16", dev), rnd(T, 24 * 128)
            return (lambda: kv.append(0, qkv, 16 * 128, 20 * 128, slots)), 0.0, T * 8 * 128 * 4
        p, w, pool = rnd(T, H * D + R + H), rnd(R), rnd(T, R)
        step = kernel.endswith("_step")
        return (lambda: K.latent_append(p[:, H * D:H * D + R], w, 1e-5, slots, pool, want_rows=not step)), 0.0, T * R * (4 if step else 6)
    if kernel.startswith("head_linear"):
        x, w, gate = rnd(T, H * (D if kernel.endswith("q") else R)), rnd(H * D, R), rnd(T, H)
        fn = (lambda: K.head_linear(x, w, H, D, R, transposed=True)) if kernel.endswith("q") else (lambda: K.head_linear(x, w, H, R, D, gate=gate))
        return fn, 2.0 * T * H * D * R, (w.numel() + T * H * (D + R)) * 2
    if kernel in ("output_norm", "layernorm"):
        x, y, w, b = rnd(T, Hd, dtype=torch.float32), rnd(T, Hd), rnd(Hd), rnd(Hd)
        if kernel == "layernorm":
            return (lambda: F.layernorm_fwd(y, w, b, 1e-5)), 0.0, T * Hd * 4
        return (lambda: K.res_norm(x, 1e-5, y=y, w_post=w, b_post=b, scale_post=w, cast=bf, kind="layer")), 0.0, T * Hd * 12
    if kernel.startswith("linear_relu2"):
        N = 8448
        x, w = rnd(T, Hd), rnd(N, Hd, scale=Hd ** -0.5)
        return (lambda: K.linear(x, w, act="relu2")), 2.0 * T * N * Hd, (w.numel() + T * (N + Hd)) * 2
    h, z, bias = rnd(T, Hd), rnd(T, E, dtype=torch.float32), rnd(E)
    if kernel.startswith("route_") or kernel == "route":
        return (lambda: M.route(z, bias, k)), 0.0, T * (E * 4 + k * 12)
    if kernel == "router_topk":
        def old():
            idx, _, _, counts, _ = M.router_topk(z, k)
            return M.Plan(idx, counts, E)
        return old, 0.0, T * (E * 8 + k * 8)
    r = M.route(z, bias, k)
    if kernel in ("moe_permute", "moe_combine"):
        idx, w, _, counts, _ = M.router_topk(z, k)

        def rows():
            pl = M.Plan(idx, counts, E)
            return pl, M.permute(h, idx, pl)
        pl, xp = rows()
        if kernel == "moe_permute":
            return rows, 0.0, T * (k + 1) * Hd * 2
        return (lambda: M.combine(xp, w, pl)), 0.0, T * (k + 1) * Hd * 2
    if kernel == "expert_rows":
        return (lambda: M.expert_rows(h, r)), 0.0, T * (k + 1) * Hd * 2
    gu, dn = rnd(E, 2 * Fh, Hd, scale=Hd ** -0.5), rnd(E, Hd, Fh, scale=Fh ** -0.5)
    xp, fl = M.expert_rows(h, r), 2.0 * T * k * 2 * Fh * Hd
    y = M.expert_linear(xp, gu, r)
    if kernel.startswith("expert_gate_up"):
        return (lambda: M.expert_linear(xp, gu, r)), fl, (gu.numel() + T * k * (Hd + 2 * Fh)) * 2
    a = M.expert_glu(y, r)
    if kernel.startswith("expert_glu"):
        return (lambda: M.expert_glu(y, r)), 0.0, T * k * Fh * 6
    if kernel.startswith("expert_down"):
        return (lambda: M.expert_linear(a, dn, r)), fl / 2, (dn.numel() + T * k * (Hd + Fh)) * 2
    o = M.expert_linear(a, dn, r)
    if kernel == "weighted_sum":
        return (lambda: M.weighted_sum(o, r, h)), 0.0, T * (k + 2) * Hd * 2
    wr, nbytes = rnd(E, Hd, scale=Hd ** -0.5), (gu.numel() + dn.numel() + 2 * T * Hd) * 2
    if kernel in ("mixture", "mixture_step"):
        def ours():
            s = M.route(K.linear(h, wr, out_dtype=torch.float32), bias, k)
            return M.weighted_sum(M.expert_linear(M.expert_glu(M.expert_linear(M.expert_rows(h, s), gu, s), s), dn, s), s)
        return ours, 1.5 * fl, nbytes
    if kernel == "moe_ffn_step":
        def theirs():
            with torch.no_grad():
                return M.moe_ffn(h, F.gemm(h, wr, out_dtype=torch.float32), gu, dn, k, True, "silu", 0.0, 0.0)
        return theirs, 1.5 * fl, nbytes
    raise SystemExit(f"Error: unknown kernel '{kernel}'")


def _build_gated(kernel, n, dev):
    """The same for attention with options (16 heads over 4 kv heads of 128; cap 50, a window of 1024 keys and 16 kept ones), gated linear
    attention (16 heads of 128 x 128) and the grouped mixture; like kernels: attention_fwd_gqa128, paged_decode, delta_*, rope_append,
    res_norm, glu_silu, route."""
    import torch

    from ..ops import functional as F
    from ..ops import moe as M
    from ..ops import stack as K
    bf = torch.bfloat16
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dtype=bf: torch.randn(*s, device=dev, generator=g).to(dtype)
    H, G, D, Hd = 16, 4, 128, 2048
    B = 1 if kernel == "gla_scan_one" else max(1, (1 << 14) // n)
    T, sc = B * n, D ** -0.5
    opt = K.HeadOptions(softcap=50.0, temp_coef=0.1, temp_every=8192) if kernel.endswith("_cap") else \
        K.HeadOptions(window=1024, keep_first=16, sink=True) if kernel.endswith("_window") else K.PLAIN
    if kernel.startswith("head_attn"):
        p = rnd(T, (2 * H + 2 * G) * D)
        q, k, v = p[:, :H * D], p[:, H * D:(H + G) * D], p[:, (H + G) * D:(H + 2 * G) * D]
        gate = p[:, (H + 2 * G) * D:] if opt.softcap else None
        keys = sum(min(i + 1, opt.window + opt.keep_first if opt.window else n) for i in range(n))
        return (lambda: K.head_attn(q, k, v, B, n, n, H, G, D, D, sc, gate, opt)), 4.0 * B * H * keys * D, T * (p.shape[1] + H * D) * 2
    if kernel.startswith("head_decode"):
        B, pages = 64, 64 * (n // 16)
        kp, vp, q, gate = rnd(pages * 16, G * D), rnd(pages * 16, G * D), rnd(B, H * D), rnd(B, H * D)
        bt = torch.randperm(pages, device=dev, generator=g).int().view(B, -1).contiguous()
        pos, keys = torch.full((B,), n - 1, dtype=torch.int32, device=dev), min(n, opt.window + opt.keep_first) if opt.window else n
        return (lambda: K.head_decode(q, kp, vp, bt, pos, H, G, D, D, sc, gate if opt.softcap else None, opt)), 4.0 * B * H * keys * D, B * keys * G * 2 * D * 2
    if kernel.startswith("gla_"):
        if kernel == "gla_step":
            B, n, T = 64, 1, 64
        p, a2, bias, w = rnd(T, 4 * H * D + 16), rnd(H * D, 16), rnd(H * D), rnd(D)
        st, sl = torch.zeros(B, H, D, D, device=dev), torch.arange(B, dtype=torch.int32, device=dev)
        if kernel == "gla_step":
            return (lambda: K.gla_step(p, a2, bias, 16.0, st, sl, w, 1e-5, B, H, D, D)), 0.0, B * H * D * D * 8
        prep = lambda: K.gla_prep(p, a2, bias, 16.0, None, B, n, H, D, D)
        if kernel == "gla_prep":
            return prep, 0.0, T * H * (3 * D * (2 + 4) + D)
        r = prep()
        return (lambda: K.gla_scan(r, st, sl, None, B, n, H, D, D, False)), 6.0 * T * H * D * D, T * H * (4 * D * 4 + D + 16)
    T = 64 if kernel.endswith("_step") else 1 << 14
    if kernel == "norm_rope_append":
        p, tab = rnd(T, (H + 2 * G) * D), F.rope_tables(64, T, device=dev)
        pos, slots, w = torch.arange(T, device=dev, dtype=torch.int32), torch.arange(T, device=dev), rnd(D)
        kp, vp = rnd(T, G * D), rnd(T, G * D)
        return (lambda: K.rope_append(p, tab, pos, H, G, D, 64, G * D, slots, kp, vp, (w, w, 1e-5))), 0.0, T * D * ((H + G) * 4 + G * 2 + G * 4)
    if kernel == "parallel_norm":
        x, y, z, w = rnd(T, Hd, dtype=torch.float32), rnd(T, Hd), rnd(T, Hd), rnd(Hd)
        return (lambda: K.res_norm(x, 1e-5, y=y, y2=z, w_pre=w, kind="plain")), 0.0, T * Hd * 14
    if kernel == "glu_gelu":
        gu = rnd(T, 2 * 5632)
        return (lambda: K.glu(gu, "gelu_tanh")), 0.0, T * 5632 * 6
    z = rnd(T, 63, dtype=torch.float32)
    route = lambda: M.route(z[:, :62], None, 6, "sigmoid", 2, 1, 1.5)
    if kernel.startswith("grouped_route"):
        return route, 0.0, T * (62 * 4 + 6 * 12)
    if kernel == "weighted_sum_gated":
        h, r = rnd(T, Hd), route()
        o = M.expert_rows(h, r)
        return (lambda: M.weighted_sum(o, r, h, z[:, 62:])), 0.0, T * 8 * Hd * 2
    raise SystemExit(f"Error: unknown kernel '{kernel}'")


def _build_streams(kernel, n, dev):
    """The same for the layers of a model with attention in chunks of 1024 keys and retention side by side (8 heads each, 2 kv heads, 128
    entries), HGRN2 (16 heads of 128 x 128) and two streams of residuals; like kernels: those of ``GATED_KERNELS``."""
    import torch

    from ..ops import functional as F
    from ..ops import moe as M
    from ..ops import stack as K
    bf = torch.bfloat16
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dtype=bf: torch.randn(*s, device=dev, generator=g).to(dtype)
    H, G, D, Hd = 8, 2, 128, 2048
    B = 1 if kernel.endswith("_one") else max(1, (1 << 14) // n)
    T, sc, opt = B * n, D ** -0.5, K.HeadOptions(chunk=1024)
    if kernel == "head_attn_chunk":
        p, sinks = rnd(T, (H + 2 * G) * D), rnd(H)
        q, k, v = p[:, :H * D], p[:, H * D:(H + G) * D], p[:, (H + G) * D:]
        keys = sum(i % opt.chunk + 1 for i in range(n))
        return (lambda: K.head_attn(q, k, v, B, n, n, H, G, D, D, sc, None, opt, 0, sinks)), 4.0 * B * H * keys * D, T * (p.shape[1] + H * D) * 2
    if kernel == "head_decode_chunk":
        B, pages = 64, 64 * (n // 16)
        kp, vp, q, sinks = rnd(pages * 16, G * D), rnd(pages * 16, G * D), rnd(B, H * D), rnd(H)
        bt = torch.randperm(pages, device=dev, generator=g).int().view(B, -1).contiguous()
        pos, keys = torch.full((B,), n - 1, dtype=torch.int32, device=dev), (n - 1) % opt.chunk + 1
        return (lambda: K.head_decode(q, kp, vp, bt, pos, H, G, D, D, sc, None, opt, sinks=sinks)), 4.0 * B * H * keys * D, B * keys * G * 2 * D * 2
    if kernel.startswith(("forget_", "retention_")):
        forget = kernel.startswith("forget_")
        H = 16 if forget else 8
        step = kernel.endswith("_step")
        if step:
            B, n, T = 64, 1, 64
        p, bias, lower, w = rnd(T, (3 if forget else 4) * H * D), rnd(H * D), torch.rand(H * D, device=dev, generator=g).to(bf), rnd(D)
        decay, tab = torch.rand(H, device=dev, generator=g) * 0.1 + 0.9, F.rope_tables(D, max(n, 2048), device=dev)
        st, sl, pos = torch.zeros(B, H, D, D, device=dev), torch.arange(B, dtype=torch.int32, device=dev), torch.arange(n, dtype=torch.int32, device=dev).repeat(B)
        if step:
            fn = (lambda: K.forget_step(p, bias, lower, st, sl, w, 1e-5, B, H, D, D)) if forget else \
                (lambda: K.retention_step(p, decay, tab, D, pos, st, sl, None, 1e-5, B, H, D, D))
            return fn, 0.0, B * H * D * D * 8
        prep = (lambda: K.forget_prep(p, bias, lower, None, B, n, H, D, D)) if forget else (lambda: K.retention_prep(p, decay, tab, D, pos, None, B, n, H, D, D))
        if kernel.endswith("_prep"):
            return prep, 0.0, T * H * (3 * D * (2 + 4) + D)
        r = prep()
        return (lambda: K.gla_scan(r, st, sl, None, B, n, H, D, D, False)), 6.0 * T * H * D * D, T * H * (4 * D * 4 + D + 16)
    T = 64 if kernel.endswith("_step") else 1 << 14
    if kernel == "unit_norm_append":
        p, pos, slots, temp = rnd(T, (H + 2 * G) * D), torch.arange(T, device=dev, dtype=torch.int32), torch.arange(T, device=dev), rnd(H)
        kp, vp = rnd(T, G * D), rnd(T, G * D)
        return (lambda: K.rope_append(p, None, pos, H, G, D, 0, G * D, slots, kp, vp, (None, None, 1e-5), temp)), 0.0, T * D * ((H + G) * 4 + G * 2 + G * 4)
    if kernel == "head_norm":
        o, w = rnd(T, 16, D, dtype=torch.float32), rnd(D)
        return (lambda: K.gated_norm(o, None, w, 1e-5, bf)), 0.0, T * 16 * D * 6
    if kernel.startswith("stream_norm"):
        S = 2
        x, y, z, w, c, m = rnd(T, S, Hd, dtype=torch.float32), rnd(T, Hd), rnd(T, Hd), rnd(Hd), rnd(S), torch.eye(S, device=dev).to(bf)
        kw = dict(y2=z, w_post=w, w_post2=w, share=0.5) if kernel.endswith("_pair") else {}
        return (lambda: K.stream_norm(x, 1e-5, y=y, mix=m, out=c, w_in=c, w_pre=w, groups=4, **kw)), 0.0, T * Hd * (S * 8 + (6 if kw else 4))
    if kernel == "glu_clamped":
        gu = rnd(T, 2 * 5632)
        return (lambda: K.glu(gu, "clamped", 7.0)), 0.0, T * 5632 * 6
    z = rnd(T, 62, dtype=torch.float32)
    r = M.route(z, None, 6, "softmax_all")
    if kernel.startswith("route_all"):
        return (lambda: M.route(z, None, 6, "softmax_all")), 0.0, T * (62 * 4 + 6 * 12)
    if kernel == "expert_glu_clamped":
        gu = rnd(r.max_rows, 2 * 704)
        return (lambda: M.expert_glu(gu, r, "clamped", 7.0)), 0.0, T * 6 * 704 * 6
    raise SystemExit(f"Error: unknown kernel '{kernel}'")


def _build(kernel, n, dev, heads=0, shape=None):
    """Returns (callable, flops, bytes) for one launch of ``kernel`` at problem size ``n``."""
    import torch

    if kernel in STACK_KERNELS:
        return _build_stack(kernel, n, dev)
    if kernel in LATENT_KERNELS:
        return _build_latent(kernel, n, dev)
    if kernel in GATED_KERNELS:
        return _build_gated(kernel, n, dev)
    if kernel in STREAM_KERNELS:
        return _build_streams(kernel, n, dev)

    from ..ops import functional as F
    bf = torch.bfloat16
    g = torch.Generator(device=dev).manual_seed(0)

    def rnd(*shape, dtype=bf, scale=1.0):
        return (torch.randn(*shape, device=dev, generator=g) * scale).to(dtype)
    if kernel == "gemm" and shape:
        # shape = (M, N, K, layout): nt = activations x weight^T (forward), nn = dgrad (weight stored [K, N]),
        # tn = wgrad (both operands stored reduction-major, fp32 accumulate)
        M, N, K, lay = shape
        if lay == "nt":
            a, b, out = rnd(M, K), rnd(N, K), torch.empty((M, N), dtype=bf, device=dev)
            return (lambda: F.gemm(a, b, out=out)), 2.0 * M * N * K, (M * K + N * K + M * N) * 2
        if lay == "nn":
            a, b, out = rnd(M, K), rnd(K, N), torch.empty((M, N), dtype=bf, device=dev)
            return (lambda: F.gemm(a, b, b_mn=True, out=out)), 2.0 * M * N * K, (M * K + N * K + M * N) * 2
        a, b, out = rnd(K, M), rnd(K, N), torch.zeros((M, N), dtype=torch.float32, device=dev)
        return (lambda: F.gemm(a, b, a_mn=True, b_mn=True, out=out, accumulate=True)), 2.0 * M * N * K, (M * K + N * K) * 2 + M * N * 8
    if kernel == "gemm":
        a, b = rnd(n, n), rnd(n, n)
        out = torch.empty((n, n), dtype=bf, device=dev)
        return (lambda: F.gemm(a, b, out=out)), 2.0 * n ** 3, 3 * n * n * 2
    if kernel == "gemm_wgrad":
        a, b = rnd(n, n), rnd(n, n)
        out = torch.zeros((n, n), dtype=torch.float32, device=dev)
        return (lambda: F.gemm(a, b, a_mn=True, b_mn=True, out=out, accumulate=True)), 2.0 * n ** 3, 2 * n * n * 2 + n * n * 8
    if kernel == "gemm_fp8":
        from ..quant import fp8
        qa, sa = fp8.quant_act_1x128(rnd(n, n))
        qb, sb = fp8.quant_weight_128x128(rnd(n, n))
        out = torch.empty((n, n), dtype=bf, device=dev)
        return (lambda: fp8.gemm_fp8(qa, sa, qb, sb, out=out)), 2.0 * n ** 3, 2 * n * n + n * n * 2
    if kernel in ("attention_fwd", "attention_bwd"):
        D, S = 64, n
        H = heads or 8
        B = max(1, (1 << 16) // S)
        qkv = rnd(B * S, 3 * H * D)
        fl = 4.0 * B * H * S * S * D / 2     # causal
        if kernel == "attention_fwd":
            return (lambda: F.attn_fwd(qkv, qkv, qkv, B, S, H, H, D, q_col0=0, k_col0=H * D, v_col0=2 * H * D)), fl, 4 * B * S * H * D * 2
        o, lse = F.attn_fwd(qkv, qkv, qkv, B, S, H, H, D, q_col0=0, k_col0=H * D, v_col0=2 * H * D)
        do, dqkv = rnd(B * S, H * D), torch.empty_like(qkv)
        return (lambda: F.attn_bwd(qkv, qkv, qkv, o, do, lse, dqkv, B, S, H, H, D, q_col0=0, k_col0=H * D, v_col0=2 * H * D)), 2.5 * fl, 8 * B * S * H * D * 2
    if kernel in ("rmsnorm", "rmsnorm_bwd"):
        T, Hd = n * 64, 1024
        x, w = rnd(T, Hd), rnd(Hd)
        if kernel == "rmsnorm":
            return (lambda: F.rmsnorm_fwd(x, w, 1e-5)), 0.0, 2 * T * Hd * 2
        y, h, rstd = F.rmsnorm_fwd(x, w, 1e-5)
        dw = torch.zeros(Hd, dtype=torch.float32, device=dev)
        return (lambda: F.rmsnorm_bwd(x, x, w, rstd, dw)), 0.0, 3 * T * Hd * 2
    if kernel == "swiglu":
        T, Fh = n * 64, 2048
        x = rnd(T, 2 * Fh)
        return (lambda: F.glu_fwd(x, "silu")), 0.0, 3 * T * Fh * 2
    if kernel == "rope":
        S, H, D = 1024, 8, 64
        B = max(1, n * 64 // S)
        x = rnd(B * S, H * D)
        cos, sin = F.rope_tables(D, S, device=dev)
        return (lambda: F.rope_(x, cos, sin, H, D, S)), 0.0, 2 * B * S * H * D * 2
    if kernel == "cross_entropy":
        T, V = n * 16, 32000
        logits = rnd(T, V)
        labels = torch.randint(0, V, (T,), device=dev)
        return (lambda: F.cross_entropy_fwd_bwd(logits, labels)), 0.0, 2 * T * V * 2
    if kernel == "adamw":
        N = n * n * 16
        p, gr = torch.randn(N, device=dev), torch.randn(N, device=dev)
        m, v, lp = torch.zeros(N, device=dev), torch.zeros(N, device=dev), torch.empty(N, dtype=bf, device=dev)
        return (lambda: F.adamw_(p, gr, m, v, lp, 1e-3, 0.9, 0.95, 1e-8, 0.01, 1)), 0.0, N * (4 * 4 + 3 * 4 + 2)
    if kernel == "paged_decode":
        from ..inference.kv_cache import PAGE, PagedKVCache
        B, Hq, Hkv, D, Lctx = 64, 32, 8, 128, n
        pages = B * (Lctx // PAGE)
        kv = PagedKVCache(1, pages, Hkv, D, "bf16", dev)
        kv.k[0].data.normal_()
        kv.v[0].data.normal_()
        bt = torch.arange(pages, device=dev, dtype=torch.int32).view(B, -1)
        sl = torch.full((B,), Lctx, dtype=torch.int32, device=dev)
        q = rnd(B, Hq * D)
        return (lambda: kv.decode(0, q, bt, sl, Hq)), 4.0 * B * Hq * Lctx * D, 2 * B * Lctx * Hkv * D * 2
    if kernel == "sampling":
        from ..inference.sampler import sample
        B, V = max(1, n // 64), 128256
        logits = rnd(B, V, dtype=torch.float32)
        t = torch.full((B,), 0.8, device=dev)
        tk = torch.full((B,), 40, dtype=torch.int32, device=dev)
        tp = torch.full((B,), 0.95, device=dev)
        return (lambda: sample(logits, t, tk, tp, seed=1, step=1)), 0.0, B * V * 4
    if kernel == "moe_ffn":
        from ..ops import moe as M
        T, Hd, Fh, E, k = n * 8, 1024, 512, 16, 2
        x, wr = rnd(T, Hd), rnd(E, Hd, scale=0.1)
        gu, dn = rnd(E, 2 * Fh, Hd, scale=0.05), rnd(E, Hd, Fh, scale=0.05)

        def run():
            with torch.no_grad():
                return M.moe_ffn(x, F.gemm(x, wr, out_dtype=torch.float32), gu, dn, k, True, "silu", 0.0, 0.0)
        return run, 2.0 * T * k * 3 * Hd * Fh, (gu.numel() + dn.numel()) * 2 + 4 * T * Hd * 2
    raise SystemExit(f"Error: unknown kernel '{kernel}' (choices: {', '.join(KERNELS)})")


def time_kernel(fn, iters=20, warmup=5, flush=True):
    """Per-launch milliseconds (list) measured with CUDA events; writes of 256 MiB evict L2 between launches (several: they
    also cover the host's time to enqueue an operator of more than one launch, which would be measured otherwise)."""
    import torch
    scrub = torch.empty(256 << 20, dtype=torch.uint8, device="cuda") if flush else None
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    out = []
    for _ in range(iters):
        if scrub is not None:
            for v in range(5):
                scrub.fill_(v)
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        out.append(e0.elapsed_time(e1))
    return out


def serve_bench(a):
    """Continuous-batching engine on a random-init preset: B requests of ``prompt_len`` random tokens, ``gen`` new tokens
    each, greedy.  Reports output tokens/s over the whole run, the median time to first token, and the mean decode step."""
    import statistics

    import torch

    from ..inference.engine import EngineConfig, InferenceEngine
    from ..inference.sampler import SamplerConfig
    from ..models.config import preset
    from ..models.dense import DenseModel
    import os
    world, rank = int(os.environ.get("WORLD_SIZE", "1")), int(os.environ.get("RANK", "0"))
    dev = torch.device("cuda", int(os.environ.get("LOCAL_RANK", "0")))
    torch.cuda.set_device(dev)
    symm = None
    if world > 1:                                  # tensor-parallel serving: one process per GPU (torch.distributed.run)
        import torch.distributed as dist

        from ..inference.tp_engine import TPInferenceEngine
        from ..parallel.symm import SymmetricHeap
        os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
        dist.init_process_group("nccl", device_id=dev)
        symm = SymmetricHeap(rank, world, dev)
    cfg = preset(a.preset)
    if a.layers > 0:
        if hasattr(cfg, "layers"):
            cfg.layers = cfg.layers[:a.layers]
        else:
            cfg.num_layers = a.layers
    if a.tp_shape > 1:
        # one rank's share of a tensor-parallel deployment, alone on this GPU: its heads, kv heads and FFN slice, the
        # replicated embedding / head, and no all-reduce - the compute side of a rank without the peers
        import dataclasses
        assert world == 1 and cfg.num_heads % a.tp_shape == 0 and cfg.ffn_hidden_size % a.tp_shape == 0
        cfg = dataclasses.replace(cfg, num_heads=cfg.num_heads // a.tp_shape, num_kv_heads=max(1, cfg.num_kv_heads // a.tp_shape),
                                  head_dim=cfg.head_dim, ffn_hidden_size=cfg.ffn_hidden_size // a.tp_shape)
    if hasattr(cfg, "num_experts"):
        from ..models.moe import MoEModel
        model = MoEModel(cfg, device=dev, dtype=torch.bfloat16, seed=0)
    elif hasattr(cfg, "architecture"):
        from ..models.registry import model_class
        model = model_class(cfg.architecture)(cfg, device=dev, dtype=torch.bfloat16, seed=0)
    else:
        model = DenseModel(cfg, device=dev, dtype=torch.bfloat16, seed=0)
    g = torch.Generator().manual_seed(0)
    if a.load == "baseline5":
        _serve_load(a, cfg, model, rank, world, symm, g)
        if world > 1:
            dist.barrier()
            symm.close()
            dist.destroy_process_group()
        return
    for B in [int(x) for x in a.batch.split(",")]:
        pages = (a.prompt_len + a.gen + 31) // 16 * B + 64
        ecfg = EngineConfig(max_batch=B, num_pages=pages, kv_mode=a.kv, weight_format=a.weights, cuda_graph=not a.no_graph,
                            enable_prefix_cache=False, max_seq_len=min(cfg.max_seq_len, a.prompt_len + a.gen + 16))
        eng = TPInferenceEngine(model, None, ecfg, rank, world, symm) if world > 1 else InferenceEngine(model, None, ecfg)
        greedy = SamplerConfig(temperature=0.0, top_k=0, top_p=1.0)
        for rep in range(3):                       # the first passes build graphs and workspaces and settle the allocator
            prompts = [torch.randint(3, cfg.vocab_size, (a.prompt_len,), generator=g).tolist() for _ in range(B)]
            torch.cuda.synchronize()
            t0 = time.perf_counter()
            reqs = [eng.add_request(p, max_tokens=a.gen, sampling=greedy) for p in prompts]
            d0 = eng.stats.decode_ms
            steps = 0
            while eng.has_pending():
                eng.step()
                steps += 1
            torch.cuda.synchronize()
            dt = time.perf_counter() - t0
        out_tokens = sum(len(r.out) for r in reqs)
        rec = {"bench": "serve", "preset": a.preset, "layers": cfg.num_layers, "batch": B, "prompt_len": a.prompt_len, "gen": a.gen, "weights": a.weights or "bf16",
               "kv": a.kv, "tp": world, "cuda_graph": eng.cfg.cuda_graph, "out_tok_s": round(out_tokens / dt, 1),
               "ttft_ms_p50": round(statistics.median((r.t_first - r.t_submit) * 1e3 for r in reqs), 2),
               "decode_ms_per_step": round((eng.stats.decode_ms - d0) / max(1, steps), 3), "total_ms": round(dt * 1e3, 1)}
        if rank == 0:
            print(json.dumps(rec), flush=True)
        del eng
        torch.cuda.empty_cache()
    if world > 1:
        dist.barrier()
        symm.close()
        dist.destroy_process_group()


def _serve_load(a, cfg, model, rank, world, symm, g):
    """Closed-loop load of BASELINE config 5: ``--requests`` (256) requests with prompt lengths uniform in
    [--prompt-min, --prompt-max] (128-2048) and ``--gen`` (256) output tokens each, ``--concurrent`` (64) in flight: a new
    request is submitted the moment one finishes.  Token ids come from the seed.  Reports output tokens/s over the whole
    run and the median / p90 time to first token (submission to first sampled token)."""
    import statistics

    import torch

    from ..inference.engine import EngineConfig, InferenceEngine
    from ..inference.sampler import SamplerConfig
    conc, nreq = a.concurrent, a.requests
    lens = torch.randint(a.prompt_min, a.prompt_max + 1, (nreq,), generator=g).tolist()
    prompts = [torch.randint(3, cfg.vocab_size, (n,), generator=g).tolist() for n in lens]
    max_len = a.prompt_max + a.gen + 16
    pages = (max_len + 15) // 16 * conc + 64
    ecfg = EngineConfig(max_batch=conc, num_pages=pages, kv_mode=a.kv, weight_format=a.weights, cuda_graph=not a.no_graph,
                        enable_prefix_cache=False, max_seq_len=min(cfg.max_seq_len, max_len))
    if world > 1:
        from ..inference.tp_engine import TPInferenceEngine
        eng = TPInferenceEngine(model, None, ecfg, rank, world, symm)
    else:
        eng = InferenceEngine(model, None, ecfg)
    greedy = SamplerConfig(temperature=0.0, top_k=0, top_p=1.0)
    # warm-up: graphs for the batch buckets, workspaces, allocator
    warm = [eng.add_request(prompts[i % nreq][:256], max_tokens=8, sampling=greedy) for i in range(conc)]
    while eng.has_pending():
        eng.step()
    del warm
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    nxt, live, done = 0, [], []
    d0, steps = eng.stats.decode_ms, 0
    while nxt < nreq or live:
        while nxt < nreq and len(live) < conc:
            live.append(eng.add_request(prompts[nxt], max_tokens=a.gen, sampling=greedy))
            nxt += 1
        eng.step()
        steps += 1
        still = []
        for r in live:
            (done if r.finished else still).append(r)
        live = still
    torch.cuda.synchronize()
    dt = time.perf_counter() - t0
    out_tokens = sum(len(r.out) for r in done)
    ttft = sorted((r.t_first - r.t_submit) * 1e3 for r in done)
    rec = {"bench": "serve_load", "load": "baseline5", "preset": a.preset, "layers": cfg.num_layers, "requests": nreq,
           "concurrent": conc, "prompt_len": [a.prompt_min, a.prompt_max], "prompt_tokens": sum(lens), "gen": a.gen,
           "weights": a.weights or "bf16", "kv": a.kv, "tp": world, "tp_shape": a.tp_shape, "cuda_graph": eng.cfg.cuda_graph,
           "out_tok_s": round(out_tokens / dt, 1), "ttft_ms_p50": round(statistics.median(ttft), 2),
           "ttft_ms_p90": round(ttft[int(0.9 * (len(ttft) - 1))], 2), "total_s": round(dt, 2), "engine_steps": steps,
           "decode_ms_per_step": round((eng.stats.decode_ms - d0) / max(1, steps), 3),
           "data": "synthetic (seeded token ids; random-init weights)"}
    if rank == 0:
        print(json.dumps(rec), flush=True)


def main(argv=None):
    ap = argparse.ArgumentParser(prog="quant_bench", description="Usage: quant_bench [--kernel <name> --size N] [--inference --model m.quant --prompt p]")
    ap.add_argument("--kernel", default="")
    add_int(ap, "--size", 1024)
    ap.add_argument("--inference", action="store_true")
    ap.add_argument("--serve", action="store_true", help="serving throughput of a random-init preset: out tok/s, TTFT, decode ms/step")
    ap.add_argument("--preset", default="llama-50m")
    ap.add_argument("--batch", default="1,8,64")
    ap.add_argument("--prompt-len", type=int, default=128)
    ap.add_argument("--gen", type=int, default=64)
    ap.add_argument("--weights", default="", help="packed weight format for --serve: int8 | int4 | mxfp8 | fp4 | ternary")
    ap.add_argument("--kv", default="bf16", help="KV cache storage for --serve: bf16 | fp8 | q4")
    ap.add_argument("--no-graph", action="store_true")
    ap.add_argument("--layers", type=int, default=0, help="--serve: override the preset's layer count (fits big shapes on one GPU)")
    ap.add_argument("--tp-shape", type=int, default=1, help="--serve on one GPU: serve one rank's share of a TP=N deployment "
                                                             "(heads and FFN divided by N, no collectives)")
    ap.add_argument("--model", default="")
    ap.add_argument("--prompt", default="test")
    add_int(ap, "--iters", 20)
    add_int(ap, "--warmup", 5)
    add_int(ap, "--heads", 0)
    ap.add_argument("--shape", default="", help="gemm only: MxNxK[:nt|nn|tn]")
    ap.add_argument("--peaks", default="")
    ap.add_argument("--json", action="store_true")
    ap.add_argument("--load", default="", help="--serve: 'baseline5' = closed-loop load (256 requests, prompts 128-2048, 256 "
                                               "outputs, 64 concurrent) instead of the fixed-batch sweep")
    ap.add_argument("--requests", type=int, default=256)
    ap.add_argument("--concurrent", type=int, default=64)
    ap.add_argument("--prompt-min", type=int, default=128)
    ap.add_argument("--prompt-max", type=int, default=2048)
    ap.add_argument("--comm", action="store_true", help="fused compute+collective kernels against NCCL + plain kernels "
                                                        "(run under torch.distributed.run; see cli/bench_comm.py)")
    ap.add_argument("--comm-ops", default="all", help="--comm: comma-separated subset of zero2, fsdp, all_reduce, tp_gemm")
    ap.add_argument("--link-gbs", type=float, default=770.0, help="--comm: NVLink bandwidth per direction per GPU, GB/s")
    ap.add_argument("--gemm-tflops", type=float, default=1382.0, help="--comm: sustained bf16 GEMM rate for the roofline")
    ap.add_argument("--zero-mb", type=int, default=256, help="--comm: flat fp32 gradient buffer of the ZeRO-2 step, MiB")
    ap.add_argument("--unit-mb", type=int, default=436, help="--comm: fp32 gradients of one FSDP unit, MiB")
    ap.add_argument("--tokens", type=int, default=8192, help="--comm: rows of the tensor-parallel products")
    ap.add_argument("--hidden", type=int, default=4096)
    ap.add_argument("--ffn", type=int, default=14336)
    ap.add_argument("--copy-ctas", type=int, default=12)
    a = ap.parse_args(argv)
    if a.comm:
        from .bench_comm import comm_bench
        comm_bench(a)
        return 0
    if a.size <= 0 or a.size > 16384:
        print("Error: --size needs 1..16384", file=sys.stderr)
        return 2
    import torch
    if a.kernel:
        if not torch.cuda.is_available():
            print("Error: kernel benchmarks need a CUDA device", file=sys.stderr)
            return 1
        groups = {"all": KERNELS, "stack": STACK_KERNELS, "latent": LATENT_KERNELS, "gated": GATED_KERNELS, "streams": STREAM_KERNELS}
        names = [n for k in a.kernel.split(",") for n in groups.get(k, (k,))]
        peaks = json.load(open(a.peaks)) if a.peaks else {}
        for name in names:
            shape = None
            if a.shape:
                dims, _, lay = a.shape.partition(":")
                shape = tuple(int(x) for x in dims.lower().split("x")) + (lay or "nt",)
            fn, flops, nbytes = _build(name, a.size, torch.device("cuda"), a.heads, shape)
            ms = time_kernel(fn, a.iters, a.warmup)
            best, med = min(ms), statistics.median(ms)
            rec = {"kernel": name, "size": a.shape or a.size, "ms_best": round(best, 5), "ms_median": round(med, 5),
                   "gbs": round(nbytes / best / 1e6, 1), "tflops": round(flops / best / 1e9, 2)}
            if peaks:
                rec["frac_hbm_of_measured"] = round(rec["gbs"] / peaks["hbm_gbs"], 3)
                if name.startswith(("delta_scan", "gla_scan", "forget_scan", "retention_scan")):      # fp32 arithmetic: against the FMA lanes at the largest clock
                    sms = torch.cuda.get_device_properties(0).multi_processor_count
                    rec["frac_fp32_fma"] = round(rec["tflops"] / (2 * FP32_FMA_PER_SM * sms * peaks.get("sm_max_mhz", 1965.0) * 1e-6), 3)
                elif flops:
                    rec["frac_bf16_of_measured"] = round(rec["tflops"] / peaks["bf16_tflops"], 3)
            print(json.dumps(rec) if a.json else "  ".join(f"{k}={v}" for k, v in rec.items()), flush=True)
    if a.serve:
        serve_bench(a)
    if a.inference:
        from ..inference.engine import EngineConfig, InferenceEngine
        from ..inference.sampler import SamplerConfig
        from ..models import registry
        from .common import load_tokenizer, model_dtype, pick_device
        dev = pick_device()
        model = registry.load_any(a.model, device=dev, dtype=model_dtype(dev))
        eng = InferenceEngine(model, load_tokenizer(a.model), EngineConfig(num_pages=1024))
        t0 = time.perf_counter()
        text, st = eng.generate_with_stats(a.prompt, min(64, model.cfg.max_seq_len - 8), SamplerConfig(0.0))
        dt = time.perf_counter() - t0
        print(f"inference: {st.generated_tokens} tokens in {dt * 1e3:.1f} ms ({st.generated_tokens / max(dt, 1e-9):.1f} tok/s, ttft {st.ttft_ms:.2f} ms)")
    return 0


if __name__ == "__main__":
    sys.exit(main())
