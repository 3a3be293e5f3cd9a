"""Figudra (attention with capped scores and gates, attention in a window with kept first tokens and a sink, gated linear attention,
grouped mixtures, parallel layers, shared tensors): every mechanism alone and the whole decoder through the engine, against the
plain statements of oracle_mixers.py.  The model-level tests run on the CPU and, marked ``gpu``, on the device in true fp32 and in
bf16."""
import json
import os
import subprocess
import sys

import pytest
import torch

import oracle_mixers as O
from transformers_fusion_b200.inference.engine import EngineConfig, InferenceEngine, Request
from transformers_fusion_b200.inference.kv_cache import PAGE
from transformers_fusion_b200.inference.sampler import SamplerConfig
from transformers_fusion_b200.models import registry
from transformers_fusion_b200.models.config import FigudraConfig
from transformers_fusion_b200.models.figudra import FigudraModel
from transformers_fusion_b200.ops import functional as F
from transformers_fusion_b200.ops import moe as X
from transformers_fusion_b200.ops import stack as K

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = SamplerConfig(temperature=0.0, top_k=0, top_p=1.0)
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
RUNS = [("cpu", "float32"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu), pytest.param(("cuda", "bfloat16"), marks=pytest.mark.gpu)]


def att(heads, kv, dim, vdim, cap, coef, every, mlp=None, scale=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 1.5 * dim ** -0.5,
                                                       "softcap": cap, "q_temp": {"coef": coef, "every": every}}}


def att2(heads, kv, dim, vdim, window, keep, rot, base=10000.0, factor=1.0, mlp=None, scale=None):
    return {"type": "attention_2", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
                                                         "mask": {"size": window, "keep_first": keep},
                                                         "rot": {"dims": rot, "base": base, "scaling": {"factor": factor}}}}


def gla(heads, dim, vdim, tau, mlp=None):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def again(layer, j):
    return dict(layer, weights_of=j)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=0, groups=1, keep=1, scale=1.0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}}
    return dict(m, shared={"ff": shared}) if shared else m


def cfg(width, vocab, layers, eps=1e-5):
    return {"architecture": "Figudra", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


G1 = gla(3, 24, 40, 7.0, moe(8, 2, 24, 56, 4, 2, 2.5))
A1 = att(6, 3, 16, 24, 9.0, 0.7, 10, moe(6, 3, 40))
CONFIGS = {
    # every kind of layer and feed-forward, a layer without one, tensors of earlier layers used again
    "mixed": cfg(96, 211, [att2(6, 2, 16, 48, 20, 5, 8, 500.0, 3.0, dense(160)), G1, A1, att(4, 4, 40, 16, 30.0, 0.25, 7), again(G1, 1), again(A1, 2)],
                 eps=1e-4),
    # sizes that fit no vector width; a window of one page exactly; all experts, one of one (a large eps: heads this small can read out
    # nearly nothing, and a norm with a small one would turn the bf16 rounding of that into anything)
    "odd": cfg(50, 101, [att(3, 1, 10, 14, 4.0, 1.0, 3, moe(3, 3, 7, 9)), att2(2, 2, 9, 7, 16, 3, 6, 100.0, 0.5, moe(1, 1, 13, 5)),
                         gla(2, 9, 7, 2.0, dense(30))], eps=0.02),
    # windows alone, so that pages go back: more kept tokens than the window, none, a page's worth and one
    "windows": cfg(64, 128, [att2(4, 4, 32, 24, 9, 20, 32, mlp=dense(96)), gla(2, 40, 12, 16.0), att2(4, 1, 16, 16, 33, 0, 2, 50.0, 4.0),
                             att2(2, 1, 24, 32, 17, 17, 12)]),
    "linear": cfg(48, 90, [gla(4, 16, 20, 1.0, dense(64)), again(gla(4, 16, 20, 1.0, dense(64)), 0), gla(2, 64, 12, 30.0)], eps=1e-6),
    # the register tiles of the device kernels: wide heads, many query heads per kv head, many experts
    "wide": cfg(256, 300, [att(8, 2, 128, 128, 40.0, 0.4, 50, dense(320)), att2(24, 2, 64, 96, 130, 7, 64, mlp=moe(40, 5, 96, 64, 5, 2, 1.5)),
                           gla(4, 128, 128, 16.0, moe(12, 1, 32, 24, 3, 1)), att(20, 1, 96, 64, 15.0, 0.3, 9), att2(4, 4, 128, 128, 70, 16, 96)]),
    # heads beyond the tensor-core forms
    "large": cfg(128, 90, [att(2, 1, 136, 24, 20.0, 0.5, 8, dense(48)), gla(1, 200, 260, 16.0), att2(3, 3, 16, 200, 40, 4, 16, mlp=moe(64, 6, 16, 0, 32, 6))]),
}
RANKS = {"mixed": 8, "odd": 5, "windows": 3, "linear": 16, "wide": 16, "large": 24}


def config(name):
    d = CONFIGS[name]
    return FigudraConfig.from_dict(d, shapes={f"l{i}.mix.a1": (RANKS[name], d["width"]) for i, l in enumerate(d["layers"])})


def build(name, device="cpu", dtype="float32", seed=0):
    """The model and its plain statement.  For bf16 the routers' choices are made clear ones (an expert that rounding swaps for
    another is a different function of the token): channel 0 of the residual is the same positive number for every token, left
    alone by all layers, and the routers see it through weights far apart."""
    m = FigudraModel(config(name), device="cpu", dtype=torch.bfloat16, seed=seed)
    if dtype == "bfloat16":
        m.tok_embeddings.data[:, 0] = 4.0
        for i, l in enumerate(m.layers):
            l.norm1.data[0] = 1.0
            l.mixer.o.data[0] = 0
            f = l.mlp
            if f is None:
                continue
            f.down.data[..., 0, :] = 0
            if hasattr(f, "router"):
                E = f.spec.experts
                f.router.data[:E].mul_(0.02)
                f.router.data[:E, 0] = (torch.randperm(E, generator=torch.Generator().manual_seed(i)) - E / 2) * (3.0 / E)
                if f.shared is not None:
                    f.shared.down.data[0] = 0
    plain = O.PlainFigudra(CONFIGS[name], {n: t.clone() for n, t in m.named_tensors()})
    out = FigudraModel(m.cfg, device=device, dtype=getattr(torch, dtype), seed=None)
    for (_, a), (_, b) in zip(out.named_tensors(), m.named_tensors()):
        a.copy_(b)
    return out, plain


def engine(m, **kw):
    base = dict(max_batch=8, num_pages=64, max_seq_len=512)
    base.update(kw)
    return InferenceEngine(m, None, EngineConfig(**base))


def toks(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def off(got, want):
    """Largest over the rows of the root mean square of the difference, in units of the logits' spread."""
    want = want.double()
    return float((got.double().cpu() - want).pow(2).mean(-1).sqrt().max() / want.std())


def limit(run):
    return {"float32": 2e-4, "bfloat16": 0.08}[run[1]]


def feed_all(eng, seq, cuts):
    """All logits of one sequence cut into the given portions."""
    r, out, at = Request([]), [], 0
    for n in cuts:
        out.append(eng.feed([(r, seq[at:at + n], list(range(n)))])[0])
        at += n
    assert at == len(seq)
    eng.end(r)
    return torch.cat(out)


def close(got, ref, tol):
    got = got.detach().cpu().double()
    assert got.isfinite().all() and float((got - ref).abs().max()) < tol * max(1.0, float(ref.abs().max()))


def types(device, fp32=1e-5, bf16=2e-2):
    return [(torch.float32, fp32)] + ([(torch.bfloat16, bf16)] if device == "cuda" else [])


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H", [96, 50, 37, 2048, 5120])
def test_embedding_norm_and_parallel_sum(device, H):
    g = torch.Generator().manual_seed(H)
    r = lambda *s: torch.randn(*s, generator=g)
    tab, y, z, we, w, ids = r(50, H), r(9, H), r(9, H), r(H), r(H), torch.randint(0, 50, (9,), generator=g)
    eps = 1e-2
    for dt, tol in types("cuda", 4e-6, 8e-3):
        c = lambda t: t.to(dt).to(device)
        q = lambda t: t.to(dt).double()
        x = torch.empty(9, H, device=device)
        a = K.res_norm(x, eps, ids=ids.to(device), table=c(tab), w_post=c(we), w_pre=c(w), kind="plain")
        first = O.plain_norm(q(tab)[ids], q(we), eps)
        close(x, first, 4e-6)                                       # 32-bit in both
        close(a, O.plain_norm(first, q(w), eps), tol)
        start = x.cpu().double()
        rows = torch.tensor([8, 3], dtype=torch.int32, device=device)
        both = start + (q(y) + q(z))
        close(K.res_norm(x, eps, y=c(y), y2=c(z), w_pre=c(w), row_index=rows, kind="plain"), O.plain_norm(both, q(w), eps)[[8, 3]], tol)
        assert torch.equal(x.cpu().double(), start)
        close(K.res_norm(x, eps, y=c(y), y2=c(z), w_pre=c(w), kind="plain"), O.plain_norm(both, q(w), eps), tol)
        close(x, both, 1e-6)
        assert K.res_norm(x, eps, y=c(y), kind="plain") is None      # a mixer alone
        close(x, both + q(y), 1e-6)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("M,N", [(5, 96), (3, 13), (200, 64)])
def test_gelu_gate(device, M, N):
    gu = torch.randn(M, 2 * N, generator=torch.Generator().manual_seed(N)) * 3
    for dt, tol in types(device, 2e-6, 1e-2):
        x = K.rows(M, 2 * N, dt, device)
        x.copy_(gu)
        u = x.cpu().double()
        close(K.glu(x, "gelu_tanh"), O.gelu_tanh(u[:, :N]) * u[:, N:], tol)


def shuffled_pages(T, seed=1, extra=3):
    n = (T + PAGE - 1) // PAGE
    order = torch.randperm(n + extra, generator=torch.Generator().manual_seed(seed))[:n]
    return order, order[torch.arange(T) // PAGE] * PAGE + torch.arange(T) % PAGE, (n + extra) * PAGE


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,G,D,V,dims,normed", [(4, 2, 32, 24, 16, 1), (3, 1, 128, 64, 128, 1), (2, 2, 96, 8, 32, 1), (5, 5, 10, 6, 6, 1), (2, 1, 200, 40, 64, 1),
                                                 (4, 2, 64, 64, 0, 1), (4, 2, 48, 16, 0, 0), (3, 1, 9, 5, 0, 0), (2, 1, 264, 16, 32, 1), (6, 2, 128, 136, 24, 1)])
def test_normed_rotation_and_append(device, H, G, D, V, dims, normed):
    T, p0, base, factor, eps = 40, 1000, 300.0, 5.0, 1e-3
    g = torch.Generator().manual_seed(D)
    order, slots, n = shuffled_pages(T)
    slots[7] = -1
    x, wq, wk = torch.randn(T, (H + G) * D + G * V + 3, generator=g), torch.rand(D, generator=g) + 0.5, torch.rand(D, generator=g) - 1.5
    tables = F.rope_tables(dims, p0 + T, base, "linear", factor, device=device) if dims else None
    for dt, tol in types(device, 2e-5, 2e-2):
        p = K.rows(T, x.shape[1], dt, device)
        p.copy_(x)
        u = p.cpu().double()
        kp, vp = torch.zeros(n, G * D, dtype=dt, device=device), torch.zeros(n, G * V, dtype=dt, device=device)
        ws = (wq.to(dt).to(device), wk.to(dt).to(device), eps) if normed else None
        K.rope_append(p, tables, torch.arange(p0, p0 + T, dtype=torch.int32, device=device), H, G, D, dims, G * V, slots.to(device), kp, vp, ws)
        q, k = u[:, :H * D].view(T, H, D), u[:, H * D:(H + G) * D].view(T, G, D)
        if normed:
            q, k = O.plain_norm(q, wq.to(dt).double(), eps), O.plain_norm(k, wk.to(dt).double(), eps)
        if dims:
            q, k = O.rotate_linear(q, p0, dims, base, factor), O.rotate_linear(k, p0, dims, base, factor)
        close(p[:, :H * D], q.reshape(T, -1), tol)
        close(p[:, H * D:(H + G) * D], k.reshape(T, -1), tol)
        assert torch.equal(p.cpu()[:, (H + G) * D:].double(), u[:, (H + G) * D:])
        keep = slots >= 0
        assert torch.equal(kp[slots[keep].to(device)].cpu(), p.cpu()[keep, H * D:(H + G) * D])
        assert torch.equal(vp[slots[keep].to(device)].cpu(), p.cpu()[keep, (H + G) * D:(H + G) * D + G * V])
        rest = torch.ones(n, dtype=torch.bool)
        rest[slots[keep]] = False
        assert not kp[rest.to(device)].any() and not vp[rest.to(device)].any()


# name -> (options of the product, options of the plain statement)
def options(window=0, keep=0, cap=0.0, sink=False, temp=(0.0, 1)):
    return (K.HeadOptions(window, keep, cap, sink, *temp),
            dict(window=window or None, keep_first=keep, cap=cap or None, sink=sink, temp=temp if temp[0] else None))


OPTIONS = {"plain": options(), "cap": options(cap=6.0), "loose cap": options(cap=80.0, temp=(0.5, 3)), "temp": options(temp=(0.8, 20)),
           "sink": options(sink=True), "window": options(window=40), "kept": options(window=70, keep=5, sink=True), "page": options(window=16, keep=17),
           "wide": options(window=128, keep=129, sink=True), "one": options(window=1, keep=1), "early": options(window=3, keep=300),
           "all": options(window=33, keep=2, cap=9.0, sink=True, temp=(0.3, 11))}


def peaks(T, window, keep):
    """(query, key) pairs that should find one another, or just not: far keys, tile and page borders, the edges of the window and of
    the first tokens that are kept."""
    out = [(T - 1, 0), (T - 2, 127), (T - 3, 128), (200, 63), (128, 127), (129, 0), (64, 15), (16, 16), (0, 0)]
    if window:
        out += [(i, i - window + e) for i in (window, window + 1, 131, 255, 257, T - 5) for e in (0, 1)]
        out += [(T - 7, keep - 1), (T - 8, keep), (window + keep + 3, keep - 1), (window + keep + 4, keep)]
    return [(i, j) for i, j in out if 0 <= j <= i < T]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("option", OPTIONS)
@pytest.mark.parametrize("H,G,D,V,T", [(3, 3, 16, 24, 150), (4, 2, 96, 128, 290), (2, 1, 128, 40, 385), (2, 2, 10, 6, 70), (1, 1, 136, 64, 90), (6, 2, 64, 64, 1)])
def test_prompt_attention(device, option, H, G, D, V, T):
    opt, plain_opt = OPTIONS[option]
    g = torch.Generator().manual_seed(D)
    q, k, v = torch.randn(T, H, D, generator=g), torch.randn(T, G, D, generator=g), torch.randn(T, G, V, generator=g)
    for i, j in peaks(T, opt.window, opt.keep_first):
        q[i] = k[j].repeat_interleave(H // G, 0) * 2.0
    gate = torch.randn(T, H * V, generator=g) * 2
    scale = 3.0 * D ** -0.5
    for dt, tol in types(device, 2e-5):
        c = lambda t: t.reshape(T, -1).to(dt)
        flat = K.rows(T, (H * D + 7) // 8 * 8 + H * V, dt, device)
        qq, gg = flat[:, :H * D], flat[:, (H * D + 7) // 8 * 8:]
        qq.copy_(c(q))
        gg.copy_(c(gate))
        kk, vv = c(k).to(device), c(v).to(device)
        u = lambda t, *s: t.to(dt).double().reshape(T, *s)
        plain = torch.stack([O.attend_options(u(q, H, D)[:, h], u(k, G, D)[:, h // (H // G)], u(v, G, V)[:, h // (H // G)], 0, scale, **plain_opt)
                             for h in range(H)], 1)
        want = plain * O.sigmoid(u(gate, H, V))
        close(K.head_attn(qq, kk, vv, 1, T, T, H, G, D, V, scale, gg, opt).reshape(T, H, V), want, tol)
        close(K.head_attn(qq, kk, vv, 1, T, T, H, G, D, V, scale, None, opt).reshape(T, H, V), plain, tol)
        for n in {(T + 2) // 3, min(T, 2)}:          # the last queries alone, without the keys that none of them sees
            lo = max(0, T - n - opt.window + 1) if opt.window else 0
            kept = min(opt.keep_first, lo)
            some = lambda t: torch.cat([t[:kept], t[lo:]])
            got = K.head_attn(qq[-n:], some(kk), some(vv), 1, n, kept + T - lo, H, G, D, V, scale, gg[-n:], opt, T - n)
            close(got.reshape(n, H, V), want[-n:], tol)
        two = lambda t: torch.cat([t, t.flip(0)])    # another sequence beside it
        ff = two(flat)
        o = K.head_attn(ff[:, :H * D], two(kk), two(vv), 2, T, T, H, G, D, V, scale, ff[:, (H * D + 7) // 8 * 8:], opt)
        close(o.reshape(2, T, H, V)[0], want, tol)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("option", OPTIONS)
@pytest.mark.parametrize("H,G,D,V", [(6, 2, 40, 24), (16, 2, 128, 128), (24, 2, 64, 96), (20, 1, 96, 64), (3, 3, 10, 6), (2, 1, 136, 200)])
def test_paged_decoding(device, option, H, G, D, V):
    """Pages in a shuffled order with others' rows between them, sequences of unequal length, several splits."""
    T = 330
    opt, plain_opt = OPTIONS[option]
    g = torch.Generator().manual_seed(D)
    order, slots, n = shuffled_pages(T)
    k, v = torch.randn(T, G, D, generator=g), torch.randn(T, G, V, generator=g)
    pairs = sorted(set(peaks(T, opt.window, opt.keep_first)))
    at = [i for i, _ in pairs]
    q = torch.stack([k[j].repeat_interleave(H // G, 0) for _, j in pairs]) * 2
    gate = torch.randn(len(at), H * V, generator=g) * 2
    scale = 3.0 * D ** -0.5
    for dt, tol in types(device, 2e-5):
        kp, vp = (torch.full((n, G * w), 9.0, dtype=dt, device=device) for w in (D, V))
        kp[slots.to(device)] = k.reshape(T, -1).to(dt).to(device)
        vp[slots.to(device)] = v.reshape(T, -1).to(dt).to(device)
        u = lambda t: t.to(dt).double()
        qd, kd, vd = u(q), u(k), u(v)
        want = torch.stack([torch.stack([O.attend_options(qd[b:b + 1, h], kd[:i + 1, h // (H // G)], vd[:i + 1, h // (H // G)], i, scale, **plain_opt)[0]
                                         for h in range(H)]) for b, i in enumerate(at)])
        qq = K.rows(len(at), H * D, dt, device)
        qq.copy_(q.reshape(len(at), -1))
        bt = order.int().to(device).repeat(len(at), 1)
        pos = torch.tensor(at, dtype=torch.int32, device=device)
        gg = gate.to(dt).to(device)
        for splits in (None, 1, 3):
            got = K.head_decode(qq, kp, vp, bt, pos, H, G, D, V, scale, None, opt, splits)
            close(got.reshape(len(at), H, V), want, tol)
        close(K.head_decode(qq, kp, vp, bt, pos, H, G, D, V, scale, gg, opt).reshape(len(at), H, V), want * O.sigmoid(u(gate).view(len(at), H, V)), tol)


def test_options_would_show():
    """Of the inputs above: one token more or less in the window or in the kept first ones, a sink left out, another cap or temperature
    change the result by far more than the limits."""
    T, D = 150, 16
    g = torch.Generator().manual_seed(D)
    q, k, v = (torch.randn(T, D, generator=g).double() for _ in range(3))
    for name, change in (("kept", dict(window=69)), ("kept", dict(window=71)), ("kept", dict(keep_first=4)), ("kept", dict(keep_first=6)),
                         ("kept", dict(sink=False)), ("all", dict(cap=10.0)), ("all", dict(temp=(0.3, 12))), ("all", dict(temp=(0.31, 11)))):
        opt = OPTIONS[name][1]
        for i, j in peaks(T, opt["window"], opt["keep_first"]):
            q[i] = k[j] * 2
        a, b = (O.attend_options(q, k, v, 0, 3.0 * D ** -0.5, **dict(opt, **c)) for c in ({}, change))
        assert float((a - b).abs().max()) > 2e-3, (name, change)


def gla_case(B, S, H, D, V, rank, seed, dt, device, spread=3.0):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    p = K.rows(B * S, 2 * H * (D + V) + rank, dt, device)
    p.copy_(r(*p.shape))
    a2 = K.padded_weight(H * D, rank, dt, device)
    a2.copy_(r(H * D, rank) * rank ** -0.5)
    bias = r(H * D) * spread
    bias[::5], bias[1::7] = 12.0, -40.0                 # channels that forget nothing, and everything
    return p, a2, bias.to(dt).to(device)


def gla_plain(p, a2, bias, tau, H, D, V, state=None):
    """Of one sequence's rows: (outputs [T, H, V], gates [T, H V], states)."""
    x, n = p.cpu().double(), H * D
    T = x.shape[0]
    q, k, v = x[:, :n].view(T, H, D) * D ** -0.5, x[:, n:2 * n].view(T, H, D), x[:, 2 * n:2 * n + H * V].view(T, H, V)
    a = O.channel_decay(x[:, 2 * n + 2 * H * V:] @ a2.cpu().double().T + bias.cpu().double(), tau).view(T, H, D)
    both = [O.gated_linear_scan(q[:, h], k[:, h], v[:, h], a[:, h], None if state is None else state[h]) for h in range(H)]
    return torch.stack([o for o, _ in both], 1), x[:, 2 * n + H * V:2 * n + 2 * H * V], torch.stack([s for _, s in both])


GLA_SIZES = [(2, 16, 24, 8, 16.0), (3, 48, 64, 16, 1.0), (1, 9, 7, 5, 0.5), (2, 128, 128, 16, 16.0), (1, 200, 136, 24, 4.0), (2, 64, 200, 3, 16.0), (1, 300, 20, 16, 8.0)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,D,V,rank,tau", GLA_SIZES)
def test_gated_linear_prompts(device, H, D, V, rank, tau):
    """Unequal sequences side by side, then their next portions from the states the first ones left."""
    B, S, first, lens = 3, 37, 21, [37, 22, 30]
    for dt, tol in types(device, 1e-5, 1e-5):                     # the recurrence is fp32 in both
        p, a2, bias = gla_case(B, S, H, D, V, rank, D + V, dt, device)
        rows = p.view(B, S, -1)
        state = torch.full((5, H, D, V), 9.0, device=device)
        slots = torch.tensor([3, 0, 4], dtype=torch.int32, device=device)
        one = lambda lo, hi, n, past: K.gla_scan(
            K.gla_prep(part(lo, hi), a2, bias, tau, n, B, hi - lo, H, D, V), state, slots, n, B, hi - lo, H, D, V, past).view(B, hi - lo, H, V)

        def part(lo, hi):
            out = K.rows(B * (hi - lo), p.shape[1], dt, device)
            out.copy_(rows[:, lo:hi].reshape(-1, p.shape[1]))
            return out
        n = torch.tensor(lens, dtype=torch.int32, device=device)
        junk = torch.full((1 << 20,), float("nan"), device=device)   # what freed memory may hold
        del junk
        whole = one(0, S, n, False)
        ends = state.clone()
        a = one(0, first, None, False)
        b = one(first, S, n - first, True)
        for i, L in enumerate(lens):
            want, _, last = gla_plain(rows[i, :L], a2, bias, tau, H, D, V)
            close(whole[i, :L], want, tol)
            assert not whole[i, L:].any()                          # padding: zeros, whatever the memory held
            close(a[i], want[:first], tol)
            close(b[i, :L - first], want[first:], tol)
            for s in (ends, state):
                close(s[slots[i]], last, tol)
        assert torch.equal(state[[1, 2]].cpu(), torch.full((2, H, D, V), 9.0))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,D,V,rank,tau", GLA_SIZES)
def test_gated_linear_step(device, H, D, V, rank, tau):
    B, eps = 3, 1e-3
    for dt, tol in types(device, 1e-5, 1e-2):
        p, a2, bias = gla_case(B, 1, H, D, V, rank, D, dt, device)
        w = (torch.rand(V, generator=torch.Generator().manual_seed(1)) + 0.5).to(dt).to(device)
        state = torch.randn(4, H, D, V, generator=torch.Generator().manual_seed(2)).to(device)
        before, slots = state.clone(), torch.tensor([2, -1, 0], dtype=torch.int32, device=device)
        got = K.gla_step(p, a2, bias, tau, state, slots, w, eps, B, H, D, V)
        for b, sl in ((0, 2), (2, 0)):
            o, gate, last = gla_plain(p[b:b + 1], a2, bias, tau, H, D, V, before[sl].cpu().double())
            want = O.plain_norm(o[0], w.cpu().double(), eps) * O.silu(gate.view(H, V))
            close(got[b].reshape(H, V), want, tol)
            close(state[sl], last, 1e-5)
        assert torch.equal(state[[1, 3]], before[[1, 3]])


@pytest.mark.parametrize("device", DEVICES)
def test_long_memory_of_the_state(device):
    """A value written at the first token and read by a key that nothing else has written, 400 tokens later."""
    S, D, V, tau = 401, 16, 8, 16.0
    x = torch.zeros(S, 2 * (D + V) + 2)
    x[0, D + 3], x[0, 2 * D:2 * D + V] = 1.0, 5.0          # k, v of the first token
    x[:, D + 4], x[:, 2 * D:2 * D + V] = 1.0, x[:, 2 * D:2 * D + V] + 1.0
    x[-1, 3] = 1.0                                         # q of the last one
    a2, bias = torch.zeros(D, 2), torch.full((D,), 8.0)
    want = gla_plain(x, a2, bias, tau, 1, D, V)[0][-1]
    assert float(want.min()) > 1.0
    c = lambda t: t.to(device)
    state, slot = torch.zeros(1, 1, D, V, device=device), torch.zeros(1, dtype=torch.int32, device=device)
    for cut in (S, 400, 6):
        out = []
        for lo, hi in ((0, cut), (cut, S)):
            if hi > lo:
                r = K.gla_prep(c(x[lo:hi]).contiguous(), c(a2), c(bias), tau, None, 1, hi - lo, 1, D, V)
                out.append(K.gla_scan(r, state, slot, None, 1, hi - lo, 1, D, V, lo > 0))
        close(torch.cat(out)[-1], want, 5e-5)                # 400 decays near one, each rounded to 2^-24


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("T,E,k,groups,keep", [(5, 6, 2, 3, 2), (300, 16, 4, 2, 1), (1, 1, 1, 1, 1), (64, 40, 5, 8, 3), (700, 300, 9, 10, 4), (3, 4, 4, 4, 4),
                                               (257, 8, 1, 8, 1), (70, 300, 40, 1, 1), (33, 32, 4, 32, 7), (40, 1024, 8, 32, 2), (9, 24, 5, 4, 4)])
def test_grouped_routing(device, T, E, k, groups, keep):
    g = torch.Generator().manual_seed(T + E)
    both = torch.randn(T, E + 1, generator=g) * 2                    # a row of the matrix behind the experts: not theirs
    both[:, E] = 50.0
    z = both[:, :E]
    z[T // 2] = 0.5                                                  # all equal: the lower group and index first
    if T > 2:
        z[0] = z[0].round()                                          # ties
    r = X.route(both.to(device)[:, :E], None, k, "sigmoid", groups, keep, 1.7)
    for t in range(T):
        want = O.route_groups(z[t].double(), k, groups, keep, 1.7)
        got = dict(zip(r.idx[t].tolist(), r.w[t].tolist()))
        if t == 0 and T > 2:                                         # marks of groups may tie but for rounding: any of them
            assert len(got) == k and abs(sum(got.values()) - 1.7) < 1e-4
            continue
        assert r.idx[t].tolist() == [e for e, _ in want]
        assert max(abs(got[e] - w) for e, w in want) < 1e-5
    rows = r.row_of.reshape(-1).tolist()
    assert len(set(rows)) == T * k and max(rows) < r.max_rows == len(r.expert_of_tile) * 128
    tile = r.expert_of_tile.tolist()
    assert all(tile[x // 128] == e for x, e in zip(rows, r.idx.reshape(-1).tolist()))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("T,H,E,k,groups,keep,F,Fs", [(5, 96, 6, 2, 2, 1, 24, 56), (70, 50, 3, 3, 1, 1, 7, 9), (300, 64, 9, 1, 3, 2, 33, 0), (1, 128, 40, 5, 10, 4, 96, 64),
                                                      (400, 96, 4, 2, 4, 2, 40, 24)])
def test_grouped_mixture(device, T, H, E, k, groups, keep, F, Fs):
    c = FigudraConfig.from_dict(cfg(H, 11, [gla(1, 8, 8, 4.0, moe(E, k, F, Fs, groups, keep, 2.5))]))
    for dt, tol in types(device):
        m = FigudraModel(c, device=device, dtype=dt, seed=T)
        h = K.rows(T, H, dt, device)
        h.copy_(torch.randn(T, H, generator=torch.Generator().manual_seed(T)))
        w = {n: t.cpu().double() for n, t in m.named_tensors()}
        p = "l0.mlp."
        three = lambda q: tuple(w[p + q + n] for n in (".gate", ".up", ".down"))
        hd = h.cpu().double()
        args = (hd, w[p + "router"], k, groups, keep, 2.5, [three(f"e{e}") for e in range(E)])
        chosen = lambda z: [[e for e, _ in O.route_groups(x, k, groups, keep, 1.0)] for x in z]
        z = hd @ w[p + "router"].T
        noise = torch.randn(z.shape, generator=torch.Generator().manual_seed(3)) * 1e-3
        clear = torch.tensor([sorted(a) == sorted(b) == sorted(d) for a, b, d in zip(chosen(z), chosen(z + noise), chosen(z - noise))])
        want = O.grouped_mixture(*args, three("shared") if Fs else None, w.get(p + "shared.sg"))
        got = m.layers[0].mlp(h, lambda x, i, n, v, act=None: K.linear(x, v.data, act=act))
        assert int(clear.sum()) >= 0.9 * T
        close(got[clear.to(device)], want[clear], tol)
        if Fs:                                         # neither the shared expert nor its gate is a rounding
            for other in (O.grouped_mixture(*args), O.grouped_mixture(*args, three("shared"), w[p + "shared.sg"] * 0)):
                assert float((other - want).abs().max()) > 5 * tol


# ------------------------------------------------------------------------------------------------ the decoder
@pytest.mark.parametrize("run", RUNS, ids=str)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(name, run):
    m, plain = build(name, *run)
    seq = toks(150, m.cfg.vocab_size)
    res, ref = [], []
    want = plain.run(seq, residuals=ref)
    got = m.head(m.hidden_states(torch.tensor([seq]), res))
    assert len(res) == len(ref) == len(m.layers)
    for a, b in zip(res, ref):
        assert a.dtype == torch.float32
        assert float((a.cpu().double() - b).pow(2).mean().sqrt() / b.pow(2).mean().sqrt()) < limit(run)
    assert off(got, want) < limit(run)
    assert off(feed_all(engine(m), seq, [150]), want) < limit(run)
    assert off(feed_all(engine(m), seq[:1], [1]), want[:1]) < limit(run)


@pytest.mark.parametrize("run", RUNS, ids=str)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_decoding_and_portions(name, run):
    """The same sequence token by token from its first token, from a prompt, and in portions of several sizes."""
    m, plain = build(name, *run, seed=1)
    n = 90
    seq = toks(n, m.cfg.vocab_size, 1)
    want = plain.run(seq)
    eng = engine(m)
    for cuts in ([1] * n, [53] + [1] * 37, [2] * 45, [16, 16, 1, 15, 17, 25], [3, 64, 2, 1, 1, 19], [33, 57], [1, 89]):
        assert off(feed_all(eng, seq, cuts), want) < limit(run), cuts
    assert eng.cache.allocator.num_free == 64 and len(eng.cache.free_slots) == 8


@pytest.mark.parametrize("run", RUNS, ids=str)
@pytest.mark.parametrize("name", ["mixed", "wide", "windows"])
def test_batches_of_unequal_requests(name, run):
    """Requests of unequal length prefilled and decoded together; some end early, their pages and slots go to new requests, and every
    position equals the request alone."""
    m, plain = build(name, *run, seed=2)
    lens, V = [1, 70, 33, 17, 2], m.cfg.vocab_size
    seqs = [toks(l + 20, V, 10 + i) for i, l in enumerate(lens)]
    want = [plain.run(s) for s in seqs]
    eng = engine(m, max_batch=5, num_pages=24)
    junk = [torch.full((n,), float("nan"), device=run[0]) for n in (1 << 12, 1 << 16, 1 << 18, 1 << 20, 1 << 24)]
    del junk                             # what freed memory may hold: padding must not bring it in
    for rep in range(2):                 # the second pass runs on pages and slots that the first one gave back
        reqs = [Request([]) for _ in seqs]
        outs = eng.feed([(r, s[:l], [l - 1] if i % 2 else list(range(l))) for i, (r, s, l) in enumerate(zip(reqs, seqs, lens))])
        for i, (o, l) in enumerate(zip(outs, lens)):
            assert off(o, want[i][l - 1:l] if i % 2 else want[i][:l]) < limit(run)
        live = list(range(len(seqs)))
        for t in range(20):
            got = eng.feed([(reqs[i], [seqs[i][lens[i] + t]], [0]) for i in live])
            for i, o in zip(live, got):
                assert off(o, want[i][lens[i] + t:lens[i] + t + 1]) < limit(run), (rep, t, i)
            if t in (4, 9, 13):
                eng.end(reqs[live.pop(t % len(live))])
        for i in live:
            eng.end(reqs[i])
        assert eng.cache.allocator.num_free == 24 and len(eng.cache.free_slots) == 5


@pytest.mark.parametrize("run", RUNS, ids=str)
@pytest.mark.parametrize("name", ["mixed", "windows"])
def test_long_decoding(name, run):
    """Through many pages; with windows alone only the kept first pages and the window's stay held."""
    m, plain = build(name, *run, seed=3)
    seq = toks(330, m.cfg.vocab_size, 3)
    want = plain.run(seq)
    eng = engine(m)
    r = Request([])
    out = [eng.feed([(r, seq[:20], list(range(20)))])[0]]
    for t in seq[20:]:
        out.append(eng.feed([(r, [t], [0])])[0])
    assert off(torch.cat(out), want) < limit(run)
    held = [p for p in r.pages if p >= 0]
    if name == "windows":
        assert eng.cache.kept_pages == 2 and len(held) <= eng.cache.pages_needed(330) == 6 and min(r.pages[:2]) >= 0 and r.pages[2:17] == [-1] * 15
    else:
        assert len(held) == 21
    assert 64 - eng.cache.allocator.num_free == len(held)
    eng.end(r)
    assert off(feed_all(eng, seq, [300] + [1] * 30), want) < limit(run)
    assert eng.cache.allocator.num_free == 64


def test_faults_would_show():
    """The fp32 limit is far below what one wrong constant, a lost tensor or gate, or a layer with its own instead of the shared state
    does to these models' logits."""
    m, plain = build("mixed", seed=1)
    seq = toks(60, m.cfg.vocab_size, 1)
    want = plain.run(seq)
    far = 20 * limit(("cpu", "float32"))
    for change in (lambda l: l[0]["mixer"]["mask"].update(size=19), lambda l: l[0]["mixer"]["mask"].update(keep_first=4), lambda l: l[0]["mixer"].update(scale=0.2),
                   lambda l: l[0]["mixer"]["rot"].update(base=400.0), lambda l: l[0]["mixer"]["rot"]["scaling"].update(factor=2.5),
                   lambda l: l[2]["mixer"].update(softcap=8.0), lambda l: l[2]["mixer"]["q_temp"].update(coef=0.6),
                   lambda l: l[3]["mixer"]["q_temp"].update(every=8), lambda l: l[1]["mixer"].update(tau=6.0),
                   lambda l: l[1]["mlp"]["router"].update(top=3), lambda l: l[1]["mlp"]["router"]["groups"].update(keep=1),
                   lambda l: l[1]["mlp"]["router"].update(scale=2.4), lambda l: l[1]["mlp"].pop("shared"), lambda l: l.pop()):
        other = json.loads(json.dumps(CONFIGS["mixed"]))
        change(other["layers"])
        assert off(O.PlainFigudra(other, plain.w).run(seq), want) > far, other
    for name, value in (("embed.norm", 1.0), ("l0.mix.q.norm", 1.0), ("l0.mix.k.norm", 1.0), ("l1.mix.norm", 1.0), ("l1.mix.a2.b", 0.0), ("l1.mix.a1", 0.0),
                        ("l1.mix.g", 0.0), ("l2.mix.g", 0.0), ("l1.mlp.shared.sg", 0.0), ("final.norm", 1.0), ("l3.norm1", 1.0)):
        w = dict(plain.w, **{name: torch.full_like(plain.w[name], value)})
        assert off(O.PlainFigudra(CONFIGS["mixed"], w).run(seq), want) > far, name


# ------------------------------------------------------------------------------------------------ scheduler
@pytest.mark.parametrize("run", RUNS[:2], ids=str)
@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("pipeline", [True, "force", False])
def test_greedy_generation(name, run, pipeline):
    """Through the scheduler: more requests than slots, unequal prompts, stop tokens seen late by the pipelined schedule."""
    m, plain = build(name, *run, seed=4)
    prompts = [toks(n, m.cfg.vocab_size, 20 + n) for n in (5, 40, 17, 1, 33)]
    want = [plain.greedy(p, 12) for p in prompts]
    eng = engine(m, max_batch=3, num_pages=40, pipeline_decode=pipeline, enable_prefix_cache=False)
    assert eng.generate_batch(prompts, 12, GREEDY) == want
    stop = want[1][3]
    r = eng.add_request(prompts[1], 12, GREEDY, stop_ids=(stop,))
    s = eng.add_request(prompts[0], 12, GREEDY)
    while eng.has_pending():
        eng.step()
    assert r.out == want[1][:want[1].index(stop) + 1] and s.out == want[0]
    assert eng.cache.allocator.num_free == 40


def test_prefixes_are_shared_without_state_or_windows():
    layers = [att(2, 1, 16, 8, 10.0, 0.5, 9, dense(40)), att(4, 2, 8, 16, 20.0, 0.5, 9)]
    d = cfg(32, 70, layers)
    m = FigudraModel(FigudraConfig.from_dict(d), seed=6)
    plain = O.PlainFigudra(d, {n: t.clone() for n, t in m.named_tensors()})
    head = toks(50, 70, 1)
    eng = engine(m, max_batch=1)
    for p in [head + toks(9, 70, 2), head + toks(30, 70, 3)]:
        assert eng.generate_batch([p], 6, GREEDY)[0] == plain.greedy(p, 6)
    assert eng.stats.prefix_hit_tokens == 48
    assert engine(build("mixed")[0]).prefix is None and engine(build("windows")[0]).prefix is None


@pytest.mark.gpu
def test_generation_bf16_gpu():
    """bf16 generation with CUDA graphs agrees with the eager passes, and its choices are near the top of the plain logits."""
    m, plain = build("wide", "cuda", "bfloat16", seed=5)
    prompts = [toks(n, 300, 30 + n) for n in (5, 140, 17)]
    a = engine(m, cuda_graph=True).generate_batch(prompts, 10, GREEDY)
    b = engine(m, cuda_graph=False).generate_batch(prompts, 10, GREEDY)
    assert a == b
    for p, o in zip(prompts, a):
        lg = plain.run(p + o)[len(p) - 1:-1]
        gap = lg.max(-1).values - lg.gather(1, torch.tensor(o)[:, None])[:, 0]
        assert float(gap.max()) < 0.5 * float(lg.std())


@pytest.mark.gpu
def test_low_bit_weights_gpu():
    m, plain = build("wide", "cuda", "bfloat16", seed=6)
    assert set(engine(m, weight_format="int8").packed) >= {"layers.0.proj", "layers.0.o", "layers.0.gate_up", "layers.1.down", "layers.2.proj"}
    seq = toks(60, 300, 6)
    assert off(feed_all(engine(m, weight_format="int8"), seq, [40] + [1] * 20), plain.run(seq)) < 0.15
    m, plain = build("mixed", "cuda", "bfloat16", seed=6)          # tensors used by two layers are packed once
    assert not any(n.startswith(("layers.4.", "layers.5.")) for n in engine(m, weight_format="int8").packed)


# ------------------------------------------------------------------------------------------------ configuration, folders, tools
def test_config_reader():
    for name, d in CONFIGS.items():
        c = config(name)
        assert c.to_dict() == d
        m = FigudraModel(c, seed=None)
        assert m.param_count() == c.num_params() == sum(t.numel() for t in m.parameters())
    c = config("mixed")
    assert c.window == 0 and c.keep_first == 5 and config("windows").window == 33 and config("windows").keep_first == 20
    assert c.active_params() != c.num_params()
    m = FigudraModel(c)
    assert m.layers[4].mixer.proj is m.layers[1].mixer.proj and m.layers[4].mixer.index == 4 and m.layers[4].mlp is m.layers[1].mlp
    for at, change, what in ((1, lambda l: l["mlp"]["router"].update(top=7), "choose 7 of 8"), (1, lambda l: l.update(type="other"), "unknown mixer"),
                             (0, lambda l: l["mlp"].update(kind="other"), "unknown feed-forward"), (0, lambda l: l["mixer"].update(kv_heads=4), "divide"),
                             (0, lambda l: l["mixer"]["rot"].update(dims=18), "rotate"), (4, lambda l: l["mixer"].update(tau=1.0), "other sizes"),
                             (4, lambda l: l.update(weights_of=9), "no tensors"), (4, lambda l: l.update(weights_of=4), "no tensors"), (2, lambda l: l["mixer"]["q_temp"].update(every=2.5), "whole")):
        bad = json.loads(json.dumps(CONFIGS["mixed"]))
        change(bad["layers"][at])
        with pytest.raises(ValueError, match=what):
            FigudraConfig.from_dict(bad)
    chain = json.loads(json.dumps(CONFIGS["mixed"]))
    chain["layers"].append(dict(chain["layers"][4], weights_of=4))
    assert FigudraConfig.from_dict(chain).layers[6].weights_of == 1


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    d = tmp_path_factory.mktemp("figudra")
    m, plain = build("mixed", seed=7)
    registry.save_folder(m, d)
    return d, plain


def test_folder_roundtrip(folder):
    """Sizes that only a tensor gives come from the folder's tensors."""
    d, plain = folder
    m = registry.load_any(d)
    assert isinstance(m, FigudraModel) and m.layers[1].mixer.spec.rank == RANKS["mixed"] == m.layers[4].mixer.spec.rank
    assert all(t.double().equal(plain.w[n]) for n, t in m.named_tensors()) and len(m.named_tensors()) == len(plain.w)


def tool(*args, stdin=None, device="cpu"):
    env = dict(os.environ, PYTHONPATH=ROOT)
    if device == "cpu":
        env["CUDA_VISIBLE_DEVICES"] = ""
    p = subprocess.run([sys.executable, "-m", "transformers_fusion_b200.cli", *map(str, args)], capture_output=True, text=True, env=env, timeout=300,
                       input=stdin)
    assert p.returncode == 0, p.stdout[-2000:] + p.stderr[-2000:]
    return p.stdout


@pytest.mark.parametrize("device", DEVICES)
def test_trace_run(folder, tmp_path, device):
    d, plain = folder
    a, b = toks(40, 211, 1), toks(9, 211, 2)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:30], "want": [0, 29]}, {"id": "y", "tokens": b[:8], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": b[8:], "want": [0]}, {"id": "x", "tokens": a[30:31], "want": [0]}], "end": ["y"]}]
    steps += [{"step": t - 29, "entries": [{"id": "x", "tokens": [a[t]], "want": [0] if t % 2 else []}], "end": ["x"] if t == 39 else []}
              for t in range(31, 40)]
    out = tool("trace_run", "--model", d, "--dtype", "float32", "--out", tmp_path, "--max-tokens", 64, "--device", device,
               stdin="".join(json.dumps(s) + "\n" for s in steps), device=device)
    assert [l for l in out.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    wa, wb = plain.run(a), plain.run(b)
    read = lambda i: torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, 211)
    assert off(read(0), wa[[0, 29]]) < 2e-4 and off(read(1), torch.stack([wb[8], wa[30]])) < 2e-4
    assert off(read(2), wa[31:32]) < 2e-4 and not (tmp_path / "3.f32").exists()


def test_tools_open_a_folder(folder):
    d, _ = folder
    out = tool("quant_info", d)
    assert "Architecture: Figudra" in out and "layer 1: gla heads=3 dim=24 vdim=40 rank=8 experts=8 top=2 ffn=24 shared=56 groups=2/4" in out
    assert "layer 0: head_attention heads=6 kv_heads=2 dim=16 vdim=48 window=20 keep_first=5 ffn=160" in out and "weights_of=1" in out
    assert "tok/s]" in tool("quant_infer", d, "hi", "--max-tokens", 4, "--seed", 3)
