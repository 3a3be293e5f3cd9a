"""Lanedra (differential window attention + gated delta rule): every mechanism alone and the whole decoder through the engine,
against the plain statements of oracle_mixers.py.  The model-level tests run on the CPU and, marked ``gpu``, on the device in
true fp32 and in bf16."""
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
from transformers_fusion_b200.models.config import LanedraConfig
from transformers_fusion_b200.models.lanedra import LanedraModel
from transformers_fusion_b200.ops import functional as F
from transformers_fusion_b200.ops import stack as K

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = SamplerConfig(temperature=0.0, top_k=0, top_p=1.0)
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
RUNS = [("cpu", "float32"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu), pytest.param(("cuda", "bfloat16"), marks=pytest.mark.gpu)]


def att(heads, kv, dim, vdim, window, diff, rot, base=10000.0, yarn=None, scale=None, kv_from=None, ff=0):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "diff": diff, "scale": scale or dim ** -0.5,
         "rot": {"dims": rot, "base": base}, "mask": {"size": window}}
    if yarn:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def delta(heads, kv, dim, vdim, conv, ff=0):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def cfg(width, vocab, layers, eps=1e-5, scale=1.0):
    return {"architecture": "Lanedra", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


YA = (4.0, 64, 8.0, 1.0)
CONFIGS = {
    # all branches: shared keys with another window, scale and diff, layers without a feed-forward, partial rotation with YaRN
    "mixed": cfg(96, 211, [delta(4, 2, 24, 40, 4, ff=160), att(6, 3, 16, 48, 20, 0.3, 12, yarn=YA),
                           att(6, 3, 16, 48, 37, 0.6, 12, yarn=YA, scale=0.5, kv_from=1, ff=112), delta(3, 3, 32, 16, 2),
                           att(6, 3, 16, 48, 5, 0.2, 12, yarn=YA, kv_from=1)], eps=1e-4, scale=1.7),
    # sizes that fit no vector width, one tap, a window of one page exactly (a large eps: heads this small can read out nearly
    # nothing, and a norm with a small one would turn the bf16 rounding of that into anything)
    "odd": cfg(50, 101, [att(2, 1, 10, 14, 16, 0.4, 6, base=500.0, ff=30), delta(2, 1, 9, 7, 1, ff=22), delta(2, 2, 12, 6, 3)], eps=0.02, scale=0.3),
    # attention alone; every head has its own keys; windows below and above a page
    "attention": cfg(64, 128, [att(4, 4, 32, 24, 9, 0.5, 32, ff=96), att(4, 4, 32, 24, 33, 0.1, 16, yarn=(0.5, 40, 4.0, 1.0))]),
    "delta": cfg(48, 90, [delta(4, 1, 16, 20, 5, ff=64), delta(2, 2, 40, 12, 3)], eps=1e-6),
    # the register tiles of the device kernels: 64 / 128-entry heads, many query heads per kv head
    "wide": cfg(256, 300, [delta(4, 4, 128, 128, 4, ff=320), att(16, 1, 64, 128, 70, 0.4, 64, yarn=YA), att(4, 2, 128, 64, 130, 0.5, 64, ff=256),
                           delta(4, 2, 64, 96, 4)]),
}


def build(name, device="cpu", dtype="float32", seed=0):
    d = CONFIGS[name]
    m = LanedraModel(LanedraConfig.from_dict(d), device="cpu", dtype=torch.bfloat16, seed=seed)
    plain = O.PlainLanedra(d, {n: t.clone() for n, t in m.named_tensors()})
    return to(m, device, dtype), plain


def to(m, device, dtype):
    out = LanedraModel(m.cfg, device=device, dtype=getattr(torch, dtype), seed=None)
    for (_, a), (_, b) in zip(out.named_tensors(), m.named_tensors()):
        a.copy_(b)
    out.finalize()
    return out


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


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("dims,dim,base,yarn", [(16, 16, 1e4, None), (12, 20, 500.0, YA), (40, 64, 1e5, (3.0, 1024, 24.0, 2.0)),
                                                (8, 8, 1e4, (0.5, 40, 4.0, 1.0)), (6, 10, 100.0, (1.0, 16, 2.0, 1.0))])
def test_rotation(dims, dim, base, yarn):
    sc = dict(zip(("factor", "original", "fast", "slow"), yarn)) if yarn else None
    n = 70
    tab = F.rope_tables(dims, n, base, "yarn" if yarn else "none", yarn[0] if yarn else 1.0, yarn[1] if yarn else 0, 1.0,
                        yarn[2] if yarn else 32.0, yarn[3] if yarn else 1.0, yarn_ramp_max=dims - 1)
    x = torch.randn(n, 3 * dim + 5)
    got = K.rope_append(x.clone(), tab, torch.arange(n, dtype=torch.int32), 2, 1, dim, dims, 5)
    want = O.rotate_rows(x[:, :3 * dim].double().view(n, 3, dim), 0, dims, base, sc)
    assert torch.allclose(got[:, :3 * dim].double().view(n, 3, dim), want, atol=1e-5)
    assert torch.equal(got[:, 3 * dim:], x[:, 3 * dim:])
    assert torch.allclose(O.rotate(x[33, :dim].double(), 33, dims, base, sc), want[33, 0])


def peaked(T, H, G, D, V, far, seed):
    """Queries and keys of a prompt in which the last query of a few positions finds key ``far`` almost alone in both maps (with
    different strength, so that the maps do not cancel)."""
    g = torch.Generator().manual_seed(seed)
    q, k, v = (torch.randn(s, generator=g) for s in ((T, H, 2, D), (T, G, 2, D), (T, G, V)))
    for i, j in far:
        for h in range(H):
            q[i, h, 0] = k[j, h // (H // G), 0] * 2.0
            q[i, h, 1] = k[j, h // (H // G), 1] * 0.5
    return q, k, v


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,G,D,V,W", [(4, 2, 16, 24, 20), (2, 1, 64, 128, 64), (6, 3, 24, 40, 1), (2, 2, 10, 6, 33), (4, 1, 128, 64, 0)])
def test_attention_window_edges(device, H, G, D, V, W):
    """Keys just inside and just outside the window, in prompts and decoded, with scores that stand out."""
    T, eps, lam, diff = 150, 1e-5, 0.45, 0.3
    w = W or 10 ** 6
    far = [(i, j) for i, j in ((149, 149 - w + 1), (148, 148 - w), (100, 101 - w), (77, 77 - w), (60, 0), (16, 0), (15, 15)) if 0 <= j <= i]
    q, k, v = peaked(T, H, G, D, V, far, seed=W)
    scale = 3.0 / math.sqrt(D)
    want = O.diff_attend(q.double(), k.double(), v.double(), H, G, scale, lam, diff, eps, W or None)
    if W:                              # a window that is one token off would show
        for w2 in (W - 1, W + 1) if W > 1 else (W + 1,):
            other = O.diff_attend(q.double(), k.double(), v.double(), H, G, scale, lam, diff, eps, w2)
            assert max(float((other - want)[i].abs().max()) for i, _ in far) > 0.05
    for dt, tol in ((torch.float32, 1e-4), (torch.bfloat16, 0.06)):
        if device == "cpu" and dt == torch.bfloat16:
            continue
        qq, kk, vv = (t.reshape(T, -1).to(device, dt) for t in (q, k, v))
        ref = want if dt == torch.float32 else O.diff_attend(*(t.cpu().double().view(s) for t, s in ((qq, q.shape), (kk, k.shape), (vv, v.shape))),
                                                             H, G, scale, lam, diff, eps, W or None)
        args = (H, G, D, V, W, scale, lam, 1 - diff, eps)
        got = K.diff_attn(qq, kk, vv, 1, T, T, *args).cpu().double().view(T, H, V)
        assert float((got - ref).abs().max()) < tol * float(ref.abs().max())
        tail = K.diff_attn(qq[-37:].contiguous(), kk, vv, 1, 37, T, *args).cpu().double().view(37, H, V)    # queries = the last positions
        assert float((tail - ref[-37:]).abs().max()) < tol * float(ref.abs().max())
        # decoding: the same rows through pages in a shuffled order
        n = (T + PAGE - 1) // PAGE
        order = torch.randperm(n + 3, generator=torch.Generator().manual_seed(1))[:n]
        slots = (order[torch.arange(T) // PAGE] * PAGE + torch.arange(T) % PAGE).to(device)
        kp = torch.full(((n + 3) * PAGE, kk.shape[1]), 7.0, dtype=dt, device=device)      # what other sequences left there
        vp = torch.full(((n + 3) * PAGE, vv.shape[1]), -9.0, dtype=dt, device=device)
        kp[slots], vp[slots] = kk, vv
        at = [i for i, _ in far] + [0, 1, 31, 32]
        bt = order.int().to(device).repeat(len(at), 1)
        for splits in (None, 1, 3):
            got = K.diff_decode(qq[at].contiguous(), kp, vp, bt, torch.tensor(at, dtype=torch.int32, device=device), *args, splits=splits)
            assert float((got.cpu().double().view(-1, H, V) - ref[at]).abs().max()) < tol * float(ref.abs().max())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,G,D,V,taps", [(4, 2, 24, 40, 4), (2, 1, 9, 7, 1), (3, 3, 32, 16, 2), (2, 2, 128, 128, 4), (4, 1, 64, 33, 3), (2, 1, 160, 64, 6),
                                          (2, 1, 64, 256, 3), (1, 1, 300, 20, 2)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_delta_rule(device, H, G, D, V, taps, dtype):
    """Convolution, gates and recurrence over prompts of unequal length in one batch, then a second portion, then single tokens,
    against one-token-at-a-time statements; histories and states land in the slots they belong to."""
    if device == "cpu" and dtype == torch.bfloat16:
        pytest.skip("the bf16 form is the device's")
    g = torch.Generator().manual_seed(D + V)
    C, B = 2 * G * D + H * V, 3
    conv = (torch.randn(C, taps, generator=g) * taps ** -0.5).to(dtype)
    A, dtb = (torch.randn(H, generator=g) - 1.5).to(dtype), (torch.randn(H, generator=g)).to(dtype)
    w = (1 + 0.3 * torch.randn(V, generator=g)).to(dtype)
    slots, nslots, eps = [4, 0, 2], 6, 1e-5
    lens = [[37, 1, 18], [2, 5, 9], [1, 1, 1], [1, 1, 1]]
    rows = [torch.randn(sum(l[b] for l in lens), C + H * V + 2 * H, generator=g).to(dtype) for b in range(B)]
    want = []
    for b in range(B):
        x = rows[b].double()
        y = {}
        for n, (lo, hi) in {"q": (0, G * D), "k": (G * D, 2 * G * D), "v": (2 * G * D, C)}.items():
            y[n], _ = O.short_conv(x[:, lo:hi], conv[lo:hi].double())
        q, k, v = O.unit(y["q"].view(-1, G, D)) * D ** -0.5, O.unit(y["k"].view(-1, G, D)), y["v"].view(-1, H, V)
        beta = torch.sigmoid(x[:, C + H * V:C + H * V + H])
        dec = torch.exp(-torch.exp(A.double()) * torch.log1p(torch.exp(x[:, C + H * V + H:] + dtb.double())))
        heads = [O.delta_scan(q[:, h * G // H], k[:, h * G // H], v[:, h], beta[:, h], dec[:, h]) for h in range(H)]
        o = O.rms(torch.stack([s[0] for s in heads], 1), eps) * w.double() * O.silu(x[:, C:C + H * V]).view(-1, H, V)
        want.append((o.reshape(-1, H * V), torch.stack([s[1] for s in heads])))
    dev = lambda t: t.to(device)
    cs = torch.full((nslots, taps - 1, C), 3.0, dtype=dtype, device=device)       # left over from other sequences
    st = torch.full((nslots, H, D, V), 5.0, device=device)
    sl = torch.tensor(slots, dtype=torch.int32, device=device)
    at = [0] * B
    for step, ln in enumerate(lens):
        S = max(ln)
        p = torch.zeros(B, S, rows[0].shape[1], dtype=dtype)
        for b in range(B):
            p[b, :ln[b]] = rows[b][at[b]:at[b] + ln[b]]
        pp = K.rows(B * S, p.shape[2], dtype, device)
        pp.copy_(p.view(B * S, -1))
        single = step >= 2
        pr = K.delta_prep(pp, dev(conv), cs, sl, dev(A), dev(dtb), None if single else torch.tensor(ln, dtype=torch.int32, device=device), B, S, G, H, D, V,
                          step > 0, step=single)
        gate = pp[:, C:C + H * V]
        if single:
            o = K.delta_step(pr, st, sl, gate, dev(w), eps, B, G, H, D, V)
        else:
            o = K.gated_norm(K.delta_scan(pr, st, sl, torch.tensor(ln, dtype=torch.int32, device=device), B, S, G, H, D, V, step > 0), gate, dev(w), eps)
        o = o.cpu().double().view(B, S, -1)
        for b in range(B):
            ref = want[b][0][at[b]:at[b] + ln[b]]
            assert not o[b, ln[b]:].any()                  # padding: zeros, whatever the memory held
            assert float((o[b, :ln[b]] - ref).abs().max()) < (1e-4 if dtype == torch.float32 else 0.01) * max(1.0, float(ref.abs().max()))
            at[b] += ln[b]
    for b, s in enumerate(slots):
        assert float((st[s].cpu().double() - want[b][1]).abs().max()) < 1e-4
        if taps > 1:
            assert torch.equal(cs[s].cpu(), rows[b][at[b] - taps + 1:at[b], :C])
    for s in set(range(nslots)) - set(slots):
        assert bool((st[s] == 5.0).all()) and bool((cs[s] == 3.0).all())


@pytest.mark.gpu
def test_delta_scan_many_sequences_gpu():
    """Enough sequences that the scan takes its wide column groups; identical sequences give identical bits, and the narrow
    groups (one sequence alone) agree."""
    B, S, G, H, D, V = 40, 53, 4, 4, 128, 128
    g = torch.Generator().manual_seed(0)
    C = 2 * G * D + H * V
    one = torch.randn(S, C + H * V + 2 * H, generator=g)
    p = one.repeat(B, 1).cuda()
    conv, A, dtb = (torch.randn(C, 4, generator=g) * 0.5).cuda(), torch.full((H,), -2.0).cuda(), torch.zeros(H).cuda()
    out = []
    for n in (B, 1):
        cs, st = torch.zeros(n, 3, C).cuda(), torch.zeros(n, H, D, V).cuda()
        sl = torch.arange(n, dtype=torch.int32).cuda()
        pr = K.delta_prep(p[:n * S], conv, cs, sl, A, dtb, None, n, S, G, H, D, V, False)
        out.append((K.delta_scan(pr, st, sl, None, n, S, G, H, D, V, False).view(n, S, H, V), st))
    assert torch.equal(out[0][0][0], out[0][0][B - 1])
    assert float((out[0][0][7] - out[1][0][0]).abs().max()) < 1e-5
    assert float((out[0][1][7] - out[1][1][0]).abs().max()) < 1e-5


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H", [96, 50, 37, 2048, 5120])
def test_norms_embedding_activation(device, H):
    g = torch.Generator().manual_seed(H)
    r = lambda *s: torch.randn(*s, generator=g)
    tab, y, w1, w2, ids = r(50, H), r(9, H), 0.3 * r(H), 0.3 * r(H), torch.randint(0, 50, (9,), generator=g)
    eps, d64 = 1e-3, lambda t: t.double()
    for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 8e-3)):
        c = lambda t: t.to(dt).to(device)
        b = lambda t: t.to(dt).double()
        x = torch.empty(9, H, device=device)
        a = K.res_norm(x, eps, ids=ids.to(device), table=c(tab), scale=0.7, w_pre=c(w1))
        ref = b(tab)[ids] * 0.7
        assert torch.allclose(x.cpu().double(), ref, atol=1e-6)
        assert float((a.cpu().double() - O.centred_norm(ref, b(w1), eps)).abs().max()) < tol * 8
        rows = torch.tensor([8, 3], dtype=torch.int32, device=device)
        ref = ref + O.centred_norm(b(y), b(w2), eps)
        last = K.res_norm(x, eps, y=c(y), w_post=c(w2), w_pre=c(w1), row_index=rows)
        assert float((last.cpu().double() - O.centred_norm(ref, b(w1), eps)[[8, 3]]).abs().max()) < tol * 8
        a = K.res_norm(x, eps, y=c(y), w_post=c(w2), w_pre=c(w1))
        assert float((x.cpu().double() - ref).abs().max()) < 1e-5          # the residual is 32-bit in both
        assert float((a.cpu().double() - O.centred_norm(ref, b(w1), eps)).abs().max()) < tol * 8
        gu = r(5, 2 * H)
        got = K.glu_silu(c(gu)).cpu().double()
        ref = O.silu(b(gu)[:, :H]) * b(gu)[:, H:]
        assert float((got - ref).abs().max()) < tol * 16


@pytest.mark.gpu
@pytest.mark.parametrize("M,N,KK", [(5, 70, 200), (130, 300, 193), (1, 512, 96), (65, 64, 17)])
def test_products_gpu(M, N, KK):
    for dt, tol in ((torch.float32, 1e-6), (torch.bfloat16, 1e-6)):
        x, w = K.rows(M, KK, dt, "cuda"), K.padded_weight(N, KK, dt, "cuda")
        x.copy_(torch.randn(M, KK))
        w.copy_(torch.randn(N, KK))
        ref = x.double() @ w.double().t()
        got = K.linear(x, w, out_dtype=torch.float32).double()
        assert float((got - ref).abs().max()) < tol * KK ** 0.5 * 20       # true fp32 accumulation, no reduced-precision inputs


@pytest.mark.gpu
@pytest.mark.parametrize("D,dims,G,V", [(56, 56, 2, 88), (40, 12, 3, 72), (10, 6, 1, 14)])
def test_rope_append_and_gather_gpu(D, dims, G, V):
    T, nq, nk = 90, 4, 2 * G
    tab = F.rope_tables(dims, 128, 1e4, "yarn", 2.0, 64, yarn_ramp_max=dims - 1)
    order = torch.randperm(10)
    slots = order[torch.arange(T) // PAGE] * PAGE + torch.arange(T) % PAGE
    slots[5] = -1
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 0.03)):
        x = torch.randn(T, (nq + nk) * D + G * V).to(dt)
        kp, vp = torch.zeros(160, nk * D, dtype=dt), torch.zeros(160, G * V, dtype=dt)
        xg, kg, vg = K.rows(T, x.shape[1], dt, "cuda"), kp.cuda(), vp.cuda()
        xg.copy_(x)
        pos = torch.arange(T, dtype=torch.int32)
        K.rope_append(x, tab, pos, nq, nk, D, dims, G * V, slots, kp, vp)
        K.rope_append(xg, tuple(t.cuda() for t in tab), pos.cuda(), nq, nk, D, dims, G * V, slots.cuda(), kg, vg)
        assert float((xg.cpu().float() - x.float()).abs().max()) < tol and float((kg.cpu().float() - kp.float()).abs().max()) < tol
        assert torch.equal(vg.cpu(), vp)
        assert torch.equal(K.gather_rows(vg, order.int().cuda(), 13, 60).cpu(), K.gather_rows(vp, order.int(), 13, 60))


# ------------------------------------------------------------------------------------------------ the decoder
@pytest.mark.parametrize("run", RUNS, ids=str)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(name, run):
    m, plain = build(name, *run)
    seq = toks(150, m.cfg.vocab_size)
    res, ref = [], []
    want = plain.run(seq, residuals=ref)
    got = m.head(m.hidden_states(torch.tensor([seq]), res))
    for a, b in zip(res, ref):
        assert a.dtype == torch.float32
        assert float((a.cpu().double() - b).pow(2).mean().sqrt() / b.pow(2).mean().sqrt()) < limit(run)
    assert off(got, want) < limit(run)
    assert off(feed_all(engine(m), seq, [150]), want) < limit(run)


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
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_batches_of_unequal_requests(name, run):
    """Requests of unequal length prefilled and decoded together; some end early, their pages and slots go to new requests, and
    every position equals the request alone."""
    m, plain = build(name, *run, seed=2)
    lens, V = [1, 70, 33, 17, 2], m.cfg.vocab_size
    seqs = [toks(l + 20, V, 10 + i) for i, l in enumerate(lens)]
    want = [plain.run(s) for s in seqs]
    eng = engine(m, max_batch=5, num_pages=24, cuda_graph=True)
    for rep in range(2):                 # the second pass runs on pages and slots the first one gave back
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
    # a sequence that starts while others run, in one call with them
    a, b = Request([]), Request([])
    eng.feed([(a, seqs[1][:70], [])])
    got = eng.feed([(a, [seqs[1][70]], [0]), (b, seqs[2][:33], [32]), ])
    assert off(got[0], want[1][70:71]) < limit(run) and off(got[1], want[2][32:33]) < limit(run)
    got = eng.feed([(b, [seqs[2][33]], [0]), (a, [seqs[1][71]], [0])])
    assert off(got[1], want[1][71:72]) < limit(run) and off(got[0], want[2][33:34]) < limit(run)


@pytest.mark.parametrize("run", RUNS, ids=str)
def test_long_decoding_keeps_a_windowful_of_pages(run):
    m, plain = build("mixed", *run, seed=3)
    seq = toks(300, m.cfg.vocab_size, 3)
    want = plain.run(seq)
    eng = engine(m, num_pages=5)         # the longest window spans 37 tokens: at most (37 - 1) // 16 + 2 pages at a time
    assert m.cfg.window == 37 and eng.cache.pages_needed(10 ** 6) == 4
    r, worst = Request([]), 0.0
    worst = off(eng.feed([(r, seq[:150], [149])])[0], want[149:150])
    for t in range(150, 300):
        worst = max(worst, off(eng.feed([(r, seq[t:t + 1], [0])])[0], want[t:t + 1]))
        assert eng.cache.allocator.num_free >= 1
    assert worst < limit(run)
    assert sum(p >= 0 for p in r.pages) <= 4


def test_window_faults_would_show():
    """The limits above are far below what a window or a rotation that is one off does to these models' logits."""
    d = CONFIGS["mixed"]
    m, plain = build("mixed", seed=1)
    seq = toks(90, m.cfg.vocab_size, 1)
    want = plain.run(seq)
    for change in (lambda c: c["layers"][1]["mixer"]["mask"].update(size=21), lambda c: c["layers"][2]["mixer"]["mask"].update(size=36),
                   lambda c: c["layers"][2]["mixer"].update(diff=0.5), lambda c: c["layers"][4]["mixer"]["mask"].update(size=4),
                   lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=3.0), lambda c: c["norm"].update(eps=1e-2)):
        other = json.loads(json.dumps(d))
        change(other)
        assert off(O.PlainLanedra(other, plain.w).run(seq), want) > 50 * limit(("cpu", "float32"))


@pytest.mark.parametrize("run", RUNS[:2], ids=str)
@pytest.mark.parametrize("name", ["mixed", "odd", "attention", "delta"])
@pytest.mark.parametrize("pipeline", [True, "force", False])
def test_greedy_generation(name, run, pipeline):
    """Through the scheduler: more requests than slots, unequal prompts, stop tokens seen late by the pipelined schedule."""
    m, plain = build(name, *run, seed=4)
    prompts = [toks(n, m.cfg.vocab_size, 20 + n) for n in (5, 40, 17, 1, 33)]
    want = [plain.greedy(p, 12) for p in prompts]
    eng = engine(m, max_batch=3, num_pages=40, pipeline_decode=pipeline)
    assert eng.prefix is None            # neither recurrent state nor a window can be shared by prompt prefix
    assert eng.generate_batch(prompts, 12, GREEDY) == want
    stop = want[1][3]
    r = eng.add_request(prompts[1], 12, GREEDY, stop_ids=(stop,))
    s = eng.add_request(prompts[0], 12, GREEDY)
    while eng.has_pending():
        eng.step()
    assert r.out == want[1][:want[1].index(stop) + 1] and s.out == want[0]
    assert eng.cache.allocator.num_free == 40 and (not eng.cache.has_state or len(eng.cache.free_slots) == 3)


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
    seq = toks(60, 300, 6)
    want = plain.run(seq)
    got = feed_all(engine(m, weight_format="int8"), seq, [40] + [1] * 20)
    assert off(got, want) < 0.15


# ------------------------------------------------------------------------------------------------ configuration, folders, tools
def test_config_reader():
    for d in CONFIGS.values():
        c = LanedraConfig.from_dict(d)
        assert c.to_dict() == d
        m = LanedraModel(c, seed=None)
        assert m.param_count() == c.num_params()
    bad = json.loads(json.dumps(CONFIGS["mixed"]))
    bad["layers"][2]["mixer"]["kv_from"] = 0
    with pytest.raises(ValueError, match="no keys and values"):
        LanedraConfig.from_dict(bad)
    bad = json.loads(json.dumps(CONFIGS["mixed"]))
    bad["layers"][1]["mixer"]["rot"]["dims"] = 18
    with pytest.raises(ValueError, match="rotate"):
        LanedraConfig.from_dict(bad)
    with pytest.raises(ValueError, match="kv_mode"):
        engine(LanedraModel(LanedraConfig.from_dict(CONFIGS["delta"])), kv_mode="fp8")


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    d = tmp_path_factory.mktemp("lanedra")
    m, plain = build("mixed", dtype="bfloat16", seed=7)
    registry.save_folder(m, d)
    return d, plain


def test_folder_roundtrip(folder, tmp_path):
    d, plain = folder
    m = registry.load_any(d)
    assert isinstance(m, LanedraModel) and {n: t.double().equal(plain.w[n]) for n, t in m.named_tensors()} == {n: True for n in plain.w}
    short = LanedraModel(LanedraConfig.from_dict(CONFIGS["mixed"]), dtype=torch.bfloat16)
    short.named_tensors = lambda: LanedraModel.named_tensors(short)[:-1]
    registry.save_folder(short, tmp_path / "short")
    with pytest.raises(KeyError, match="head missing"):
        registry.load_folder(tmp_path / "short")
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.model_class("Nothing")


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
    assert "Architecture: Lanedra" in out and "layer 2: attention" in out and "kv_from=1" in out
    out = tool("quant_infer", d, "hi", "--max-tokens", 4, "--seed", 3)
    assert "tok/s]" in out
