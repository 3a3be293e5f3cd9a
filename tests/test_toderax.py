"""Toderax (chunked attention and retention side by side, HGRN2, clamped experts, norms in groups, streams of residuals): every mechanism
alone and the whole decoder through the engine, against the plain statements of oracle_mixers.py.  The model-level tests run on the CPU
and, marked ``gpu``, on the device in true fp32 and in bf16."""
import json
import math
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
from transformers_fusion_b200.models.config import ToderaxConfig
from transformers_fusion_b200.models.stack import MixerPair
from transformers_fusion_b200.models.toderax import ToderaxModel
from transformers_fusion_b200.ops import functional as F
from transformers_fusion_b200.ops import moe as X
from transformers_fusion_b200.ops import stack as K

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = SamplerConfig(temperature=0.0, top_k=0, top_p=1.0)
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
RUNS = [("cpu", "float32"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu), pytest.param(("cuda", "bfloat16"), marks=pytest.mark.gpu)]


def pair(left, right, mlp=None):
    """left: heads, kv heads, dim, vdim, chunk[, scale]; right: dim, vdim, decays, rotated entries[, base]."""
    h, g, d, v, size = left[:5]
    a = {"heads": h, "kv_heads": g, "dim": d, "vdim": v, "mask": {"size": size}, "scale": left[5] if len(left) > 5 else 1.7 * d ** -0.5}
    b = {"heads": len(right[2]), "dim": right[0], "vdim": right[1], "decay": list(right[2]), "rot": {"dims": right[3], "base": right[4] if len(right) > 4 else 300.0}}
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": a, "right": b}}


def hgrn2(heads, dim, vdim, mlp=None):
    return {"type": "hgrn2", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def moe(experts, top, ff, limit, shared=0, shared_limit=0.0):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    return dict(m, shared={"ff": shared, "limit": shared_limit}) if shared else m


def cfg(width, vocab, layers, groups=3, streams=2, eps=1e-5, scale=2.5):
    return {"architecture": "Toderax", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps, "groups": groups}, "streams": streams,
            "vocab": vocab, "width": width}


CONFIGS = {
    # chunks of unequal sizes (one of them no multiple of a page), a layer without a feed-forward, one without a shared expert
    "mixed": cfg(96, 211, [pair((6, 2, 16, 40, 24), (24, 32, (0.9, 0.99, 0.5), 16), moe(8, 3, 24, 0.6, 56, 0.9)), hgrn2(3, 24, 40, moe(6, 2, 40, 1.0)),
                           pair((4, 4, 40, 16, 37), (16, 24, (0.97, 1.0), 16, 50.0)), hgrn2(2, 16, 24)], eps=1e-4),
    # sizes that fit no vector width; chunks of one and of three positions; one expert; a single stream
    "odd": cfg(50, 101, [pair((3, 1, 9, 7, 3), (10, 6, (0.8,), 6), moe(3, 3, 7, 0.4, 9, 2.0)), hgrn2(2, 9, 7, moe(1, 1, 13, 0.7, 5, 0.3)),
                         pair((2, 2, 10, 14, 1), (7, 9, (0.6, 0.95), 2, 20.0))], groups=5, streams=1, eps=0.02, scale=1.0),
    "chunks": cfg(64, 128, [pair((4, 1, 32, 24, 16), (40, 12, (0.99, 0.9), 32), moe(4, 1, 32, 1.0, 24, 1.0)), pair((4, 4, 16, 16, 48), (16, 40, (0.95,), 0)),
                            pair((2, 1, 24, 32, 33), (8, 8, (0.7, 0.8, 0.9), 8))], groups=1, streams=3),
    "recurrent": cfg(48, 90, [hgrn2(4, 16, 20, moe(5, 4, 24, 0.8, 32, 0.5)), hgrn2(2, 64, 12)], groups=4, streams=5, eps=1e-6),
    # the register tiles of the device kernels: wide heads, many query heads per kv head, many experts
    "wide": cfg(256, 300, [pair((8, 2, 128, 128, 130, 0.2), (128, 128, (0.999, 0.9), 64, 10000.0), moe(40, 5, 96, 1.0, 64, 0.7)), hgrn2(2, 128, 128, moe(12, 1, 32, 0.8)),
                           pair((20, 1, 96, 64, 50), (64, 96, (0.99, 0.97, 0.5), 64))], groups=8, streams=4),
    # heads beyond the tensor-core forms and the register tiles
    "large": cfg(128, 90, [pair((2, 1, 136, 24, 40, 0.3), (200, 260, (0.98,), 100), moe(70, 6, 16, 0.9)), hgrn2(1, 300, 36), hgrn2(1, 40, 264)], groups=2),
}


def build(name, device="cpu", dtype="float32", seed=0):
    """The model and its plain statement.  For bf16 the routers' choices are made clear ones (an expert that rounding swaps for another is a
    different function of the token): channel 0 of every stream is one and the same positive number for every token, no layer adds to it,
    and the routers see it through weights far apart."""
    m = ToderaxModel(ToderaxConfig.from_dict(CONFIGS[name]), device="cpu", dtype=torch.bfloat16, seed=seed)
    for l in m.layers:                       # temperatures of both signs, sinks that weigh as much as a chunk
        if isinstance(l.mixer, MixerPair):
            l.mixer.left.temp.data[-1] *= -1
            l.mixer.left.sink.data.mul_(20)
    if dtype == "bfloat16":
        m.tok_embeddings.data[:, 0] = 3.0
        for i, l in enumerate(m.layers):
            for hc in l.hc:
                hc.mix.data.abs_()
                hc.read.data.abs_()
            for n in l.vector_names():
                l.vector(n)[0] = 1.0
            for t in (l.mixer.left_o, l.mixer.right_o) if isinstance(l.mixer, MixerPair) else (l.mixer.o,):
                t.data[0] = 0
            f = l.mlp
            if f is None:
                continue
            f.down.data[..., 0, :] = 0
            E = f.spec.experts
            f.router.data.mul_(0.02)
            f.router.data[:, 0] = (torch.randperm(E, generator=torch.Generator().manual_seed(i)) - E / 2) * (3.0 / E)
            if f.shared is not None:
                f.shared.down.data[0] = 0
    plain = O.PlainToderax(CONFIGS[name], {n: t.clone() for n, t in m.named_tensors()})
    out = ToderaxModel(m.cfg, device=device, dtype=getattr(torch, dtype), seed=None)
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
    return {"float32": 2e-4, "bfloat16": 0.1}[run[1]]


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
@pytest.mark.parametrize("H,groups,S", [(96, 4, 2), (50, 5, 3), (37, 1, 1), (2048, 8, 2), (5120, 1, 4), (5120, 16, 5), (768, 3, 16), (24, 24, 2)])
def test_streams_and_group_norm(device, H, groups, S):
    n, eps = 9, 1e-2
    g = torch.Generator().manual_seed(H + S)
    r = lambda *s: torch.randn(*s, generator=g)
    tab, y, z, w, wa, wb, mix, out, read, ids = r(50, H), r(n, H), r(n, H), r(H), r(H), r(H), r(S, S), r(S), r(S), torch.randint(0, 50, (n,), generator=g)
    for dt, tol in types("cuda", 1e-5, 1e-2):
        c, q = (lambda t: t.to(dt).to(device)), (lambda t: t.to(dt).double())
        x = torch.empty(n, S, H, device=device)
        a = K.stream_norm(x, eps, ids=ids.to(device), table=c(tab), scale=2.5, w_in=c(read), w_pre=c(w), groups=groups)
        xs = [q(tab)[ids] * 2.5] * S
        streams = lambda xs: torch.stack(xs, 1)
        close(x, streams(xs), 4e-6)                                  # 32-bit in both
        close(a, O.group_norm(O.streams_in(xs, q(read)), q(w), groups, eps), tol)
        x.copy_(r(n, S, H))                                          # streams that differ
        xs = list(x.cpu().double().unbind(1))
        start = x.clone()
        for kw, inner in ((dict(y=c(y)), q(y)), (dict(y=c(y), y2=c(z), w_post=c(wa), w_post2=c(wb), share=0.5),
                                                  (O.plain_norm(q(y), q(wa), eps) + O.plain_norm(q(z), q(wb), eps)) / 2)):
            x.copy_(start)
            after = O.streams_out(xs, inner, q(mix), q(out))
            rows = torch.tensor([8, 3], dtype=torch.int32, device=device)
            last = K.stream_norm(x, eps, mix=c(mix), out=c(out), w_pre=c(w), groups=groups, row_index=rows, **kw)
            close(last, O.group_norm(sum(after), q(w), groups, eps)[[8, 3]], tol)
            assert torch.equal(x, start)
            a = K.stream_norm(x, eps, mix=c(mix), out=c(out), w_in=c(read), w_pre=c(w), groups=groups, **kw)
            close(a, O.group_norm(O.streams_in(after, q(read)), q(w), groups, eps), tol)
            close(x, streams(after), 4e-6)
            x.copy_(start)
            assert K.stream_norm(x, eps, mix=c(mix), out=c(out), **kw) is None
            close(x, streams(after), 4e-6)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("M,N", [(5, 96), (3, 13), (200, 64)])
def test_clamped_gate(device, M, N):
    gu = torch.randn(M, 2 * N, generator=torch.Generator().manual_seed(N)) * 3
    gu[0, :2] = torch.tensor([-200.0, 200.0])
    for dt, tol in types(device, 2e-6, 1e-2):
        x = K.rows(M, 2 * N, dt, device)
        x.copy_(gu)
        u = x.cpu().double()
        eye = torch.eye(N, dtype=torch.float64)
        both = torch.cat([eye, 0 * eye], 1), torch.cat([0 * eye, eye], 1)
        close(K.glu(x, "clamped", 1.25), O.clamped_glu(u, both[0], both[1], eye, 1.25), tol)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("M,K_,N", [(1, 64, 48), (5, 50, 13), (16, 256, 100), (40, 96, 33), (300, 128, 260), (200, 30, 7)])
def test_product_with_bias(device, M, K_, N):
    g = torch.Generator().manual_seed(M)
    x, w, b = torch.randn(M, K_, generator=g), torch.randn(N, K_, generator=g) * K_ ** -0.5, torch.randn(N, generator=g) * 4
    for dt, tol in types(device):
        xx, ww = K.rows(M, K_, dt, device), K.padded_weight(N, K_, dt, device)
        xx.copy_(x)
        ww.copy_(w)
        bb = b.to(dt).to(device)
        close(K.linear(xx, ww, bias=bb), xx.cpu().double() @ ww.cpu().double().T + bb.cpu().double(), tol)


def shuffled_pages(T, seed=1, extra=3):
    n = (T + PAGE - 1) // PAGE
    order = torch.randperm(n + extra, generator=torch.Generator().manual_seed(seed))[:n]
    return order, order[torch.arange(T) // PAGE] * PAGE + torch.arange(T) % PAGE, (n + extra) * PAGE


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,G,D,V,dims", [(4, 2, 32, 24, 0), (3, 1, 128, 64, 0), (2, 2, 48, 8, 32), (5, 5, 10, 6, 0), (2, 1, 200, 40, 64), (3, 1, 9, 5, 0), (2, 1, 264, 16, 0)])
def test_weightless_norm_and_head_factors(device, H, G, D, V, dims):
    T, eps = 40, 1e-3
    g = torch.Generator().manual_seed(D)
    order, slots, n = shuffled_pages(T)
    slots[7] = -1
    x, temp = torch.randn(T, (H + G) * D + G * V, generator=g), torch.randn(H, generator=g)
    tables = F.rope_tables(dims, T, 100.0, device=device) if dims else None
    for dt, tol in types(device, 2e-5, 2e-2):
        p = K.rows(T, x.shape[1], dt, device)
        p.copy_(x)
        u = p.cpu().double()
        kp, vp = torch.zeros(n, G * D, dtype=dt, device=device), torch.zeros(n, G * V, dtype=dt, device=device)
        tt = temp.to(dt).to(device)
        K.rope_append(p, tables, torch.arange(T, dtype=torch.int32, device=device), H, G, D, dims, G * V, slots.to(device), kp, vp, (None, None, eps), tt)
        q, k = O.rms(u[:, :H * D].view(T, H, D), eps) * tt.cpu().double()[:, None], O.rms(u[:, H * D:(H + G) * D].view(T, G, D), eps)
        if dims:
            q, k = O.rotate_linear(q, 0, dims, 100.0), O.rotate_linear(k, 0, dims, 100.0)
        close(p[:, :H * D], q.reshape(T, -1), tol)
        close(p[:, H * D:(H + G) * D], k.reshape(T, -1), tol)
        keep = slots >= 0
        assert torch.equal(kp[slots[keep].to(device)].cpu(), p.cpu()[keep, H * D:(H + G) * D])
        assert torch.equal(vp[slots[keep].to(device)].cpu(), p.cpu()[keep, (H + G) * D:(H + G) * D + G * V])


CHUNKS = (1, 16, 24, 64, 100, 128, 130, 256, 1000)


def peaks(T, size):
    """(query, key) pairs that should find one another, or just not: the ends of chunks, far keys, tile and page borders."""
    out = [(T - 1, 0), (T - 2, 127), (T - 3, 128), (200, 63), (128, 127), (129, 0), (64, 15), (16, 16), (0, 0)]
    for c in (1, 2, T // size):
        at = c * size
        out += [(at, at - 1), (at, at), (at + 1, at - 1), (at + size - 1, at), (at + size - 2, at - 1), (at - 1, at - size)]
    return sorted({i: j for i, j in out if 0 <= j <= i < T}.items())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("size", CHUNKS)
@pytest.mark.parametrize("H,G,D,V,T", [(3, 3, 16, 24, 150), (4, 2, 96, 128, 290), (2, 1, 48, 64, 600), (2, 2, 10, 6, 70), (1, 1, 136, 64, 90), (6, 2, 64, 64, 1)])
def test_chunked_prompt_attention(device, size, H, G, D, V, T):
    g = torch.Generator().manual_seed(D)
    q, k, v = torch.randn(T, H, D, generator=g), torch.randn(T, G, D, generator=g), torch.randn(T, G, V, generator=g)
    for i, j in peaks(T, size):
        q[i] = k[j].repeat_interleave(H // G, 0) * 2.0
    sinks = torch.randn(H, generator=g) * 3
    sinks[0] = 60.0 if T == 150 else -60.0           # far above all scores, and far below
    scale, opt = 3.0 * D ** -0.5, K.HeadOptions(chunk=size)
    for dt, tol in types(device, 2e-5):
        c = lambda t: t.reshape(T, -1).to(dt).to(device)
        qq = K.rows(T, H * D, dt, device)
        qq.copy_(c(q))
        kk, vv, ss = c(k), c(v), sinks.to(dt).to(device)
        u = lambda t, *s: t.to(dt).double().reshape(T, *s)
        plain = lambda sink: torch.stack([O.attend_chunk(u(q, H, D)[:, h], u(k, G, D)[:, h // (H // G)], u(v, G, V)[:, h // (H // G)], 0, scale, size,
                                                         sinks.to(dt).double()[h] if sink else None) for h in range(H)], 1)
        want = plain(True)
        close(K.head_attn(qq, kk, vv, 1, T, T, H, G, D, V, scale, None, opt, 0, ss).reshape(T, H, V), want, tol)
        close(K.head_attn(qq, kk, vv, 1, T, T, H, G, D, V, scale, None, opt).reshape(T, H, V), plain(False), tol)
        for n in {(T + 2) // 3, min(T, 2)}:          # the last queries alone, without the chunks that none of them sees
            lo = (T - n) // size * size
            got = K.head_attn(qq[-n:], kk[lo:], vv[lo:], 1, n, T - lo, H, G, D, V, scale, None, opt, T - n, ss)
            close(got.reshape(n, H, V), want[-n:], tol)
        two = lambda t: torch.cat([t, t.flip(0)])    # another sequence beside it
        o = K.head_attn(two(qq), two(kk), two(vv), 2, T, T, H, G, D, V, scale, None, opt, 0, ss)
        close(o.reshape(2, T, H, V)[0], want, tol)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("size", CHUNKS)
@pytest.mark.parametrize("H,G,D,V", [(6, 2, 40, 24), (16, 2, 128, 128), (20, 1, 96, 64), (3, 3, 10, 6), (2, 1, 136, 200)])
def test_chunked_paged_decoding(device, size, H, G, D, V):
    T = 330
    g = torch.Generator().manual_seed(D)
    order, slots, n = shuffled_pages(T)
    k, v = torch.randn(T, G, D, generator=g), torch.randn(T, G, V, generator=g)
    pairs = peaks(T, size)
    at = [i for i, _ in pairs]
    q = torch.stack([k[j].repeat_interleave(H // G, 0) for _, j in pairs]) * 2
    sinks = torch.randn(H, generator=g) * 3
    sinks[0], scale, opt = 60.0, 3.0 * D ** -0.5, K.HeadOptions(chunk=size)
    for dt, tol in types(device, 2e-5):
        kp, vp = (torch.full((n, G * w), 9.0, dtype=dt, device=device) for w in (D, V))
        kp[slots.to(device)] = k.reshape(T, -1).to(dt).to(device)
        vp[slots.to(device)] = v.reshape(T, -1).to(dt).to(device)
        u = lambda t: t.to(dt).double()
        plain = lambda sink: torch.stack([torch.stack([O.attend_chunk(u(q)[b:b + 1, h], u(k)[:i + 1, h // (H // G)], u(v)[:i + 1, h // (H // G)], i, scale, size,
                                                                      u(sinks)[h] if sink else None)[0] for h in range(H)]) for b, i in enumerate(at)])
        qq = K.rows(len(at), H * D, dt, device)
        qq.copy_(q.reshape(len(at), -1))
        bt, pos, ss = order.int().to(device).repeat(len(at), 1), torch.tensor(at, dtype=torch.int32, device=device), sinks.to(dt).to(device)
        for splits in (None, 1, 3):
            got = K.head_decode(qq, kp, vp, bt, pos, H, G, D, V, scale, None, opt, splits, ss)
            close(got.reshape(len(at), H, V), plain(True), tol)
        close(K.head_decode(qq, kp, vp, bt, pos, H, G, D, V, scale, None, opt).reshape(len(at), H, V), plain(False), tol)


@pytest.mark.parametrize("device", DEVICES)
def test_kept_first_keys_with_chunks(device):
    """The options combine: a chunk, and the first tokens of the sequence besides."""
    T, H, D, V, size, keep, scale = 200, 2, 32, 16, 48, 5, 0.3
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(T, H, w, generator=g) for w in (D, D, V))
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    ok = (j <= i) & ((i // size == j // size) | (j < keep))
    opt = K.HeadOptions(keep_first=keep, chunk=size)
    order, slots, n = shuffled_pages(T)
    for dt, tol in types(device, 2e-5):
        u, c = (lambda t: t.to(dt).double()), (lambda t: t.reshape(T, -1).to(dt).to(device))
        want = torch.stack([torch.softmax((u(q)[:, h] @ u(k)[:, h].T * scale).masked_fill(~ok, -math.inf), -1) @ u(v)[:, h] for h in range(H)], 1)
        close(K.head_attn(c(q), c(k), c(v), 1, T, T, H, H, D, V, scale, None, opt).reshape(T, H, V), want, tol)
        kp, vp = torch.zeros(n, H * D, dtype=dt, device=device), torch.zeros(n, H * V, dtype=dt, device=device)
        kp[slots.to(device)], vp[slots.to(device)] = c(k), c(v)
        at = [3, 47, 48, 52, 150, 199]
        got = K.head_decode(c(q)[at], kp, vp, order.int().to(device).repeat(len(at), 1), torch.tensor(at, dtype=torch.int32, device=device), H, H, D, V, scale,
                            None, opt)
        close(got.reshape(len(at), H, V), want[at], tol)


def test_chunk_faults_would_show():
    """Of the inputs above: a chunk of one position more or less, chunks counted from another start, a sink left out or scaled change the
    result by far more than the limits."""
    T, D, size = 150, 16, 24
    g = torch.Generator().manual_seed(D)
    q, k, v = (torch.randn(T, D, generator=g).double() for _ in range(3))
    for i, j in peaks(T, size):
        q[i] = k[j] * 2
    run = lambda size=size, sink=1.5, pos0=0: O.attend_chunk(q, k, v, pos0, 3.0 * D ** -0.5, size, torch.tensor(sink).double() if sink is not None else None)
    for change in (dict(size=23), dict(size=25), dict(sink=None), dict(sink=1.5 * 3 * D ** -0.5)):
        assert float((run(**change) - run()).abs().max()) > 1e-2, change


# ------------------------------------------------------------------------------------------------ recurrences
def rows_of(B, S, width, seed, dt, device):
    p = K.rows(B * S, width, dt, device)
    p.copy_(torch.randn(B * S, width, generator=torch.Generator().manual_seed(seed)))
    return p


class Forget:
    """HGRN2 as the tests drive it: rows q | f | v."""
    gated = False

    def __init__(self, H, D, V, dt, device):
        g = torch.Generator().manual_seed(D + V)
        bias, lower = torch.randn(H * D, generator=g) * 3, torch.rand(H * D, generator=g)
        bias[::5], bias[1::7], lower[::3], lower[1::9] = 12.0, -40.0, 0.0, 1.0           # channels that forget all or nothing
        self.args = tuple(t.to(dt).to(device) for t in (bias, lower))
        self.sizes, self.width = (H, D, V), 2 * H * D + H * V

    def prep(self, p, lens, B, S, pos0):
        return K.forget_prep(p, *self.args, lens, B, S, *self.sizes)

    def step(self, p, state, slots, w, eps, B, pos):
        return K.forget_step(p, *self.args, state, slots, w, eps, B, *self.sizes)

    def plain(self, p, pos0=0, state=None):
        """Of one sequence's rows: outputs [T, H, V] and states."""
        (H, D, V), x, n = self.sizes, p.cpu().double(), self.sizes[0] * self.sizes[1]
        q, v = O.silu(x[:, :n]).view(-1, H, D), x[:, 2 * n:].view(-1, H, V)
        f = O.forget_gate(x[:, n:2 * n] + self.args[0].cpu().double(), self.args[1].cpu().double()).view(-1, H, D)
        both = [O.hgrn2_scan(q[:, h], f[:, h], v[:, h], None if state is None else state[h]) for h in range(H)]
        return torch.stack([o for o, _ in both], 1), torch.stack([s for _, s in both])


class Retain:
    """Retention: rows q | k | v | gate."""
    gated = True

    def __init__(self, H, D, V, dt, device, base=300.0):
        self.dims, self.base, self.device = D if D in (64, 128) else D // 4 * 2, base, device
        self.decay = torch.linspace(0.4, 1.0, H) if H > 1 else torch.tensor([0.96875])
        self.args = (self.decay.to(device), F.rope_tables(self.dims, 2000, base, device=device) if self.dims else None, self.dims)
        self.sizes, self.width = (H, D, V), 2 * H * (D + V)

    def prep(self, p, lens, B, S, pos0):
        return K.retention_prep(p, *self.args, torch.arange(pos0, pos0 + S, dtype=torch.int32, device=self.device).repeat(B), lens, B, S, *self.sizes)

    def step(self, p, state, slots, w, eps, B, pos):
        return K.retention_step(p, *self.args, torch.tensor(pos, dtype=torch.int32, device=self.device), state, slots, w, eps, B, *self.sizes)

    def plain(self, p, pos0=0, state=None):
        (H, D, V), x, n = self.sizes, p.cpu().double(), self.sizes[0] * self.sizes[1]
        q, k = (O.rotate_linear(x[:, i * n:(i + 1) * n].reshape(-1, H, D), pos0, self.dims, self.base) for i in (0, 1))
        v = x[:, 2 * n:2 * n + H * V].reshape(-1, H, V)
        both = [O.retention_scan(q[:, h], k[:, h] * D ** -0.5, v[:, h], float(self.decay[h].double()), None if state is None else state[h]) for h in range(H)]
        return torch.stack([o for o, _ in both], 1), torch.stack([s for _, s in both])


LINEAR_SIZES = [(2, 16, 24), (3, 48, 64), (1, 9, 7), (2, 128, 128), (1, 200, 136), (2, 64, 200), (1, 300, 20), (2, 6, 33)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("kind", [Forget, Retain])
@pytest.mark.parametrize("H,D,V", LINEAR_SIZES)
def test_recurrent_prompts(device, kind, H, D, V):
    """Unequal sequences side by side, then their next portions from the states the first ones left."""
    B, S, first, lens = 3, 37, 21, [37, 22, 30]
    for dt, tol in types(device, 2e-5, 2e-5):                     # the recurrence is fp32 in both
        m = kind(H, D, V, dt, device)
        p = rows_of(B, S, m.width, D, dt, device)
        rows = p.view(B, S, -1) if p.is_contiguous() else p.reshape(B, S, -1)
        state = torch.full((5, H, D, V), 9.0, device=device)
        slots = torch.tensor([3, 0, 4], dtype=torch.int32, device=device)

        def one(lo, hi, n, past):
            part = K.rows(B * (hi - lo), m.width, dt, device)
            part.copy_(rows[:, lo:hi].reshape(-1, m.width))
            return K.gla_scan(m.prep(part, n, B, hi - lo, lo), state, slots, n, B, hi - lo, H, D, V, past).view(B, hi - lo, H, V)
        n = torch.tensor(lens, dtype=torch.int32, device=device)
        junk = torch.full((1 << 20,), float("nan"), device=device)   # what freed memory may hold
        del junk
        whole = one(0, S, n, False)
        ends = state.clone()
        a = one(0, first, None, False)
        b = one(first, S, n - first, True)
        for i, L in enumerate(lens):
            want, last = m.plain(rows[i, :L])
            close(whole[i, :L], want, tol)
            assert not whole[i, L:].any()                          # padding: zeros, whatever the memory held
            close(a[i], want[:first], tol)
            close(b[i, :L - first], want[first:], tol)
            for s in (ends, state):
                close(s[slots[i]], last, tol)
        assert torch.equal(state[[1, 2]].cpu(), torch.full((2, H, D, V), 9.0))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("kind", [Forget, Retain])
@pytest.mark.parametrize("H,D,V", LINEAR_SIZES)
def test_sequences_in_segments(device, kind, H, D, V):
    """Segments of a sequence side by side: as many as fit or more, sequences that end in the first, in the middle and at the end of one,
    fresh ones and ones that go on, in slots and without."""
    B, S, lens = 4, 100, [100, 5, 48, 81]
    for dt, tol in types(device, 2e-5, 2e-5):
        m = kind(H, D, V, dt, device)
        p = rows_of(B, S, m.width, D, dt, device)
        rows = p.reshape(B, S, -1)
        slots, n = torch.tensor([3, 0, 4, -1], dtype=torch.int32, device=device), torch.tensor(lens, dtype=torch.int32, device=device)
        begin = torch.randn(5, H, D, V, generator=torch.Generator().manual_seed(5)).to(device)
        for past in (False, True):
            want = [m.plain(rows[i, :L], 0, begin[slots[i]].cpu().double() if past and slots[i] >= 0 else None) for i, L in enumerate(lens)]
            for segments in (1, 2, 3, 7, 30):
                state = begin.clone()
                got = K.gla_scan(m.prep(p, n, B, S, 0), state, slots, n, B, S, H, D, V, past, segments).view(B, S, H, V)
                for i, L in enumerate(lens):
                    close(got[i, :L], want[i][0], tol)
                    assert not got[i, L:].any()
                    if slots[i] >= 0:
                        close(state[slots[i]], want[i][1], tol)
                assert torch.equal(state[[1, 2]], begin[[1, 2]])


@pytest.mark.parametrize("device", DEVICES)
def test_long_sequence_in_segments(device):
    """Of the kernel's own choice, against the sequence in one piece."""
    H, D, V, S = 2, 32, 16, 1500
    for kind in (Forget, Retain):
        m = kind(H, D, V, torch.float32, device)
        p = rows_of(1, S, m.width, 1, torch.float32, device)
        state, slot = torch.zeros(1, H, D, V, device=device), torch.zeros(1, dtype=torch.int32, device=device)
        want, last = m.plain(p)
        for segments in (None, 1):
            close(K.gla_scan(m.prep(p, None, 1, S, 0), state, slot, None, 1, S, H, D, V, False, segments), want, 2e-5)
            close(state[0], last, 2e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("kind", [Forget, Retain])
@pytest.mark.parametrize("H,D,V", LINEAR_SIZES)
def test_recurrent_step(device, kind, H, D, V):
    B, eps, pos = 3, 1e-3, [700, 0, 5]
    for dt, tol in types(device, 1e-5, 1e-2):
        m = kind(H, D, V, dt, device)
        p = rows_of(B, 1, m.width, D, dt, device)
        w = (torch.rand(V, generator=torch.Generator().manual_seed(1)) + 0.5).to(dt).to(device)
        for weight in (w, None):
            state = torch.randn(4, H, D, V, generator=torch.Generator().manual_seed(2)).to(device)
            before, slots = state.clone(), torch.tensor([2, -1, 0], dtype=torch.int32, device=device)
            got = m.step(p, state, slots, weight, eps, B, pos)
            for b, sl in ((0, 2), (2, 0)):
                o, last = m.plain(p[b:b + 1], pos[b], before[sl].cpu().double())
                want = O.rms(o[0], eps) * (1.0 if weight is None else w.cpu().double())
                if m.gated:
                    want = want * O.silu(p[b, -H * V:].cpu().double().view(H, V))
                close(got[b].reshape(H, V), want, tol)
                close(state[sl], last, 1e-5)
            assert torch.equal(state[[1, 3]], before[[1, 3]])


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("gate,weight", [(True, True), (True, False), (False, True), (False, False)])
def test_head_norms(device, gate, weight):
    T, H, V = 11, 3, 40
    g = torch.Generator().manual_seed(3)
    o, gt, w = torch.randn(T, H, V, generator=g), torch.randn(T, H * V, generator=g), torch.randn(V, generator=g)
    for dt, tol in types(device, 1e-5, 1e-2):
        got = K.gated_norm(o.to(device), gt.to(dt).to(device) if gate else None, w.to(dt).to(device) if weight else None, 1e-2, dt)
        want = O.rms(o.double(), 1e-2) * (w.to(dt).double() if weight else 1.0) * (O.silu(gt.to(dt).double()).view(T, H, V) if gate else 1.0)
        assert got.dtype == dt
        close(got.reshape(T, H, V), want, tol)


@pytest.mark.parametrize("device", DEVICES)
def test_long_memory_of_the_states(device):
    """A value written at the first token and read 400 tokens later, by a key that nothing else has written or through gates that close."""
    S, D, V = 401, 16, 8
    r = Retain(1, D, V, torch.float32, device)
    r.decay = torch.tensor([1 - 2.0 ** -11])
    r.args = (r.decay.to(device), None, 0)
    r.dims = 0
    x = torch.zeros(S, r.width)
    x[:, 2 * D:2 * D + V], x[:, D + 4], x[-1, 3] = 1.0, 1.0, 1.0
    x[0, D + 3], x[0, D + 4], x[0, 2 * D:2 * D + V] = 4.0, 0.0, 20.0
    f = Forget(1, D, V, torch.float32, device)
    f.args = (torch.zeros(D, device=device), torch.full((D,), 1 - 2.0 ** -11, device=device))
    y = torch.zeros(S, f.width)
    y[:, D:2 * D] = -30.0                                  # every gate at its lower bound, then one value written at once
    y[0, 2 * D:] = 20000.0
    y[-1, :D] = 1.0
    for m, z in ((r, x), (f, y)):
        want = m.plain(z)[0][-1]
        assert float(want.abs().min()) > 1.0
        state, slot = torch.zeros(1, 1, D, V, device=device), torch.zeros(1, dtype=torch.int32, device=device)
        for cut in (S, 400, 6):
            out = []
            for lo, hi in ((0, cut), (cut, S)):
                if hi > lo:
                    out.append(K.gla_scan(m.prep(z[lo:hi].to(device).contiguous(), None, 1, hi - lo, lo), state, slot, None, 1, hi - lo, 1, D, V, lo > 0))
            close(torch.cat(out)[-1], want, 5e-5)          # 400 decays near one, each rounded to 2^-24


# ------------------------------------------------------------------------------------------------ mixture
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("T,E,k", [(5, 6, 2), (300, 16, 4), (1, 1, 1), (64, 40, 5), (700, 300, 9), (3, 4, 4), (257, 8, 1), (70, 300, 40), (33, 100, 4)])
def test_routing_over_all_experts(device, T, E, k):
    g = torch.Generator().manual_seed(T + E)
    z = torch.randn(T, E, generator=g) * 2
    z[T // 2] = 0.5                                                  # all equal: the lower index first
    r = X.route(z.to(device), None, k, "softmax_all")
    for t in range(T):
        want = O.route_all(z[t].double(), k)
        assert r.idx[t].tolist() == [e for e, _ in want]
        assert max(abs(a - w) for a, (_, w) in zip(r.w[t].tolist(), want)) < 1e-6
    rows, tile = r.row_of.reshape(-1).tolist(), r.expert_of_tile.tolist()
    assert len(set(rows)) == T * k and all(tile[x // 128] == e for x, e in zip(rows, r.idx.reshape(-1).tolist()))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("T,H,E,k,F,Fs", [(5, 96, 6, 2, 24, 56), (70, 50, 3, 3, 7, 9), (300, 64, 9, 1, 33, 0), (1, 128, 40, 5, 96, 64)])
def test_clamped_mixture(device, T, H, E, k, F, Fs):
    c = ToderaxConfig.from_dict(cfg(H, 11, [hgrn2(1, 8, 8, moe(E, k, F, 0.7, Fs, 1.1))], groups=1))
    for dt, tol in types(device):
        m = ToderaxModel(c, device=device, dtype=dt, seed=T)
        h = K.rows(T, H, dt, device)
        h.copy_(torch.randn(T, H, generator=torch.Generator().manual_seed(T)))
        w = {n: t.cpu().double() for n, t in m.named_tensors()}
        p = "l0.mlp."
        three = lambda q: tuple(w[p + q + n] for n in (".gate", ".up", ".down"))
        hd = h.cpu().double()
        run = lambda limit=0.7, shared_limit=1.1, shared=Fs: O.clamped_mixture(hd, w[p + "router"], k, [three(f"e{e}") for e in range(E)], limit,
                                                                             three("shared") if shared else None, shared_limit)
        chosen = lambda z: [[e for e, _ in O.route_all(x, k)] for x in z]
        z = hd @ w[p + "router"].T
        noise = torch.randn(z.shape, generator=torch.Generator().manual_seed(3)) * 1e-3
        clear = torch.tensor([sorted(a) == sorted(b) == sorted(d) for a, b, d in zip(chosen(z), chosen(z + noise), chosen(z - noise))])
        want = run()
        got = m.layers[0].mlp(h, lambda x, i, n, v, act=None: K.linear(x, v.data, act=act))
        assert int(clear.sum()) >= 0.9 * T
        close(got[clear.to(device)], want[clear], tol)
        for other in [run(limit=0.8)] + ([run(shared=0), run(shared_limit=1.2)] if Fs else []):
            assert float((other - want).abs().max()) > 1e-3


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
    for cuts in ([1] * n, [48] + [1] * 42, [2] * 45, [16, 16, 1, 15, 17, 25], [3, 64, 2, 1, 1, 19], [24, 13, 53], [1, 89]):
        assert off(feed_all(eng, seq, cuts), want) < limit(run), cuts
    assert eng.cache.allocator.num_free == 64 and (not eng.cache.has_state or len(eng.cache.free_slots) == 8)


@pytest.mark.parametrize("run", RUNS, ids=str)
@pytest.mark.parametrize("name", ["mixed", "wide", "chunks"])
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
@pytest.mark.parametrize("name", ["mixed", "chunks"])
def test_long_decoding(name, run):
    """Through many pages and chunks; pages of chunks that no layer looks at any more go back."""
    m, plain = build(name, *run, seed=3)
    seq = toks(330, m.cfg.vocab_size, 3)
    want = plain.run(seq)
    eng = engine(m)
    r = Request([])
    out = [eng.feed([(r, seq[:20], list(range(20)))])[0]]
    for i, t in enumerate(seq[20:], 21):
        out.append(eng.feed([(r, [t], [0])])[0])
        first = min(i // c * c for c in ((16, 48, 33) if name == "chunks" else (24, 37)))
        assert [p >= 0 for p in r.pages] == [k >= first // PAGE for k in range((i + PAGE - 1) // PAGE)]
        assert 64 - eng.cache.allocator.num_free == sum(p >= 0 for p in r.pages) <= eng.cache.pages_needed(330)
    assert off(torch.cat(out), want) < limit(run)
    eng.end(r)
    assert off(feed_all(eng, seq, [300] + [1] * 30), want) < limit(run)
    assert eng.cache.allocator.num_free == 64


def test_faults_would_show():
    """The fp32 limit is far below what one wrong constant, a lost tensor or a lost stream does to the model's logits."""
    m, plain = build("mixed", seed=1)
    seq = toks(60, m.cfg.vocab_size, 1)
    want = plain.run(seq)
    far = 20 * limit(("cpu", "float32"))
    left, right = (lambda l, i=0: l[i]["mixer"]["left"]), (lambda l, i=0: l[i]["mixer"]["right"])
    for change in (lambda l: left(l)["mask"].update(size=23), lambda l: left(l)["mask"].update(size=25), lambda l: left(l, 2).update(scale=0.3),
                   lambda l: right(l)["rot"].update(base=250.0), lambda l: right(l)["rot"].update(dims=14), lambda l: right(l).update(decay=[0.9, 0.98, 0.5]),
                   lambda l: l[0]["mlp"]["router"].update(top=2), lambda l: l[0]["mlp"]["expert"].update(limit=0.7),
                   lambda l: l[0]["mlp"]["shared"].update(limit=1.0), lambda l: l[0]["mlp"].pop("shared"), lambda l: l.pop()):
        other = json.loads(json.dumps(CONFIGS["mixed"]))
        change(other["layers"])
        assert off(O.PlainToderax(other, plain.w).run(seq), want) > far, other
    for change in (dict(embedding={"scale": 2.4}), dict(norm={"eps": 1e-4, "groups": 1}), dict(norm={"eps": 1e-2, "groups": 3})):
        assert off(O.PlainToderax(dict(CONFIGS["mixed"], **change), plain.w).run(seq), want) > far, change
    for name, value in (("l0.mix.left.q.b", 0.0), ("l0.mix.left.k.b", 0.0), ("l0.mix.left.v.b", 0.0), ("l0.mix.left.temp", 1.0), ("l0.mix.left.sink", 0.0),
                        ("l0.mix.left.out", 1.0), ("l2.mix.right.out", 1.0), ("l0.mix.right.g", 0.0), ("l1.mix.f.b", 0.0), ("l1.mix.lower", 0.0),
                        ("l1.mix.norm", 1.0), ("l3.norm1", 1.0), ("l0.norm2", 1.0), ("final.norm", 1.0), ("l1.hc2.in", 0.5), ("l1.hc2.out", 1.0)):
        w = dict(plain.w, **{name: torch.full_like(plain.w[name], value)})
        assert off(O.PlainToderax(CONFIGS["mixed"], w).run(seq), want) > far, name
    w = dict(plain.w, **{"l2.hc1.mix": plain.w["l2.hc1.mix"].T})
    assert off(O.PlainToderax(CONFIGS["mixed"], w).run(seq), want) > far


# ------------------------------------------------------------------------------------------------ scheduler
@pytest.mark.parametrize("run", RUNS[:2], ids=str)
@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("pipeline", [True, "force", False])
def test_greedy_generation(name, run, pipeline):
    """Through the scheduler: more requests than slots, unequal prompts, stop tokens seen late by the pipelined schedule."""
    m, plain = build(name, *run, seed=4)
    prompts = [toks(n, m.cfg.vocab_size, 20 + n) for n in (5, 40, 17, 1, 33)]
    want = [plain.greedy(p, 12) for p in prompts]
    eng = engine(m, max_batch=3, num_pages=40, pipeline_decode=pipeline)
    assert eng.prefix is None                            # state, and pages that go back
    assert eng.generate_batch(prompts, 12, GREEDY) == want
    stop = want[1][3]
    r = eng.add_request(prompts[1], 12, GREEDY, stop_ids=(stop,))
    s = eng.add_request(prompts[0], 12, GREEDY)
    while eng.has_pending():
        eng.step()
    assert r.out == want[1][:want[1].index(stop) + 1] and s.out == want[0]
    assert eng.cache.allocator.num_free == 40


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
    eng = engine(m, weight_format="int8")
    assert set(eng.packed) >= {"layers.0.proj", "layers.0.left_o", "layers.0.right_o", "layers.0.gate_up", "layers.0.down", "layers.1.proj", "layers.1.o"}
    seq = toks(60, 300, 6)
    assert off(feed_all(eng, seq, [40] + [1] * 20), plain.run(seq)) < 0.2


# ------------------------------------------------------------------------------------------------ configuration, folders, tools
def test_config_reader():
    for name, d in CONFIGS.items():
        c = ToderaxConfig.from_dict(d)
        assert c.to_dict() == d
        m = ToderaxModel(c, seed=None)
        assert m.param_count() == c.num_params() >= c.active_params()
    c = ToderaxConfig.from_dict(CONFIGS["mixed"])
    assert c.window == 37 and ToderaxConfig.from_dict(CONFIGS["recurrent"]).window == 0
    for at, change, what in ((0, lambda l: l["mlp"]["router"].update(top=9), "choose 9 of 8"), (1, lambda l: l.update(type="other"), "unknown mixer"),
                             (0, lambda l: l["mlp"].update(kind="other"), "unknown feed-forward"), (0, lambda l: l["mixer"]["left"].update(kv_heads=4), "divide"),
                             (0, lambda l: l["mixer"]["right"]["rot"].update(dims=26), "rotate"), (0, lambda l: l["mixer"]["right"].update(decay=[0.5]), "decays"),
                             (0, lambda l: l["mixer"]["left"]["mask"].update(size=0), "chunk"), (1, lambda l: l["mixer"].update(dim=513), "512")):
        bad = json.loads(json.dumps(CONFIGS["mixed"]))
        change(bad["layers"][at])
        with pytest.raises(ValueError, match=what):
            ToderaxConfig.from_dict(bad)
    for change, what in ((dict(streams=17), "streams"), (dict(norm={"eps": 1e-5, "groups": 5}), "groups")):
        with pytest.raises(ValueError, match=what):
            ToderaxConfig.from_dict(dict(CONFIGS["mixed"], **change))


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    d = tmp_path_factory.mktemp("toderax")
    m, plain = build("mixed", seed=7)
    registry.save_folder(m, d)
    return d, plain


def test_folder_roundtrip(folder):
    d, plain = folder
    m = registry.load_any(d)
    assert isinstance(m, ToderaxModel)
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
    assert "Architecture: Toderax" in out and "layer 1: hgrn2 heads=3 dim=24 vdim=40 experts=6 top=2 ffn=40" in out
    assert "layer 0: head_attention heads=6 kv_heads=2 dim=16 vdim=40 chunk=24 + retention heads=3 dim=24 vdim=32 experts=8 top=3 ffn=24 shared=56" in out
    assert "tok/s]" in tool("quant_infer", d, "hi", "--max-tokens", 4, "--seed", 3)
