"""Tekenex (latent attention, dense and mixture-of-experts feed-forwards, norms on the sublayers' outputs): every mechanism alone and
the whole decoder through the engine, against the plain statements of oracle_mixers.py.  The model-level tests run on the CPU
and, marked ``gpu``, on the device in true fp32 and in bf16."""
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
from transformers_fusion_b200.models.config import TekenexConfig
from transformers_fusion_b200.models.tekenex import TekenexModel
from transformers_fusion_b200.ops import moe as X
from transformers_fusion_b200.ops import stack as K

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = SamplerConfig(temperature=0.0, top_k=0, top_p=1.0)
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
RUNS = [("cpu", "float32"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu), pytest.param(("cuda", "bfloat16"), marks=pytest.mark.gpu)]


def layer(heads, dim, vdim, rank, mlp=None, scale=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale or dim ** -0.5}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return dict(m, shared={"ff": shared}) if shared else m


def cfg(width, vocab, layers, eps=1e-5):
    return {"architecture": "Tekenex", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


CONFIGS = {
    # every kind of feed-forward, sizes that differ from layer to layer, another scale
    "mixed": cfg(96, 211, [layer(3, 16, 48, 40, moe(6, 2, 24, 56)), layer(5, 32, 8, 24, dense(160), scale=0.31), layer(2, 48, 72, 88),
                           layer(4, 24, 24, 56, moe(5, 3, 40))], eps=1e-4),
    # sizes that fit no vector width; all experts chosen, one of one chosen
    "odd": cfg(50, 101, [layer(3, 10, 14, 22, moe(3, 3, 7, 9)), layer(1, 9, 7, 5, dense(30)), layer(2, 6, 11, 33, moe(1, 1, 13))], eps=3e-3),
    # the register tiles of the device kernels: wide latents, many heads, many experts
    "wide": cfg(256, 300, [layer(16, 128, 128, 512, moe(40, 5, 96, 64)), layer(40, 24, 40, 200, dense(320)), layer(20, 64, 96, 256, moe(9, 1, 32))]),
    # heads and latents beyond the tensor-core forms
    "large": cfg(128, 90, [layer(2, 136, 24, 72, dense(48)), layer(3, 16, 200, 520, moe(4, 2, 16))]),
}


def build(name, device="cpu", dtype="float32", seed=0):
    """The model and its plain statement.  For bf16 the routers' choices are made clear ones (an expert that rounding swaps for
    another is a different function of the token): biases far apart, small weights."""
    d = CONFIGS[name]
    m = TekenexModel(TekenexConfig.from_dict(d), device="cpu", dtype=torch.bfloat16, seed=seed)
    if dtype == "bfloat16":
        for i, l in enumerate(m.layers):
            if hasattr(l.mlp, "router"):
                E = l.mlp.spec.experts
                l.mlp.router.data.mul_(0.05)
                l.mlp.router_bias.data.copy_(torch.randperm(E, generator=torch.Generator().manual_seed(i)) * 0.6)
    plain = O.PlainTekenex(d, {n: t.clone() for n, t in m.named_tensors()})
    out = TekenexModel(m.cfg, device=device, dtype=getattr(torch, dtype), seed=None)
    for (_, a), (_, b) in zip(out.named_tensors(), m.named_tensors()):
        a.copy_(b)
    return out, plain


def engine(m, **kw):
    base = dict(max_batch=8, num_pages=64, max_seq_len=512, enable_prefix_cache=False)
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


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H", [96, 50, 37, 2048, 5120])
def test_output_norm_scale_and_residual(device, H):
    g = torch.Generator().manual_seed(H)
    r = lambda *s: torch.randn(*s, generator=g)
    tab, y, w, b, ls, wf, bf, ids = r(50, H), r(9, H) + 3, r(H), r(H), r(H), r(H), r(H), torch.randint(0, 50, (9,), generator=g)
    eps = 1e-2
    for dt, tol in ((torch.float32, 4e-6), (torch.bfloat16, 8e-3)):
        c = lambda t: t.to(dt).to(device)
        q = lambda t: t.to(dt).double()
        x = torch.empty(9, H, device=device)
        a = K.res_norm(x, eps, ids=ids.to(device), table=c(tab), cast=dt, kind="layer")
        assert torch.equal(x.cpu().double(), q(tab)[ids]) and torch.equal(a.cpu(), tab.to(dt)[ids])
        post = dict(y=c(y), w_post=c(w), b_post=c(b), scale_post=c(ls), kind="layer")
        ref = q(tab)[ids] + O.layer_norm(q(y), q(w), q(b), eps) * q(ls)
        rows = torch.tensor([8, 3], dtype=torch.int32, device=device)
        close(K.res_norm(x, eps, w_pre=c(wf), b_pre=c(bf), row_index=rows, **post), O.layer_norm(ref, q(wf), q(bf), eps)[[8, 3]], tol)
        assert torch.equal(x.cpu().double(), q(tab)[ids])
        a = K.res_norm(x, eps, cast=dt, **post)
        assert float((x.cpu().double() - ref).abs().max()) < 1e-4 and x.dtype == torch.float32      # 32-bit in both
        assert torch.equal(a.cpu(), x.cpu().to(dt)) and a.data_ptr() != x.data_ptr()
        z = x.clone()
        assert K.res_norm(z, eps, **post) is None
        close(z, ref + (ref - q(tab)[ids]), 2e-6 if dt == torch.float32 else 1e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("M,N,KK", [(5, 70, 200), (130, 300, 193), (3, 512, 2048), (64, 48, 1100)])
def test_squared_relu_product(device, M, N, KK):
    g = torch.Generator().manual_seed(M)
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
        if device == "cpu" and dt == torch.bfloat16:
            continue
        x, w = K.rows(M, KK, dt, device), K.padded_weight(N, KK, dt, device)
        x.copy_(torch.randn(M, KK, generator=g))
        w.copy_(torch.randn(N, KK, generator=g) * KK ** -0.5)
        z = x.cpu().double() @ w.cpu().double().T
        close(K.linear(x, w, act="relu2"), O.relu2(z), tol)
        zz = K.linear(x, w)
        close(K.activation(zz, "relu2"), O.relu2(zz.cpu().double()), 1e-2 if dt == torch.bfloat16 else 1e-6)


def peaked(T, H, D, V, far, seed):
    """Queries and keys of a prompt in which the query of a few positions finds one key almost alone in every head."""
    g = torch.Generator().manual_seed(seed)
    q, k, v = (torch.randn(s, generator=g) for s in ((T, H, D), (T, H, D), (T, H, V)))
    for i, j in far:
        q[i] = k[j] * 2.0
    return q, k, v


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,G,D,V,T", [(3, 3, 16, 24, 150), (2, 2, 64, 128, 300), (2, 1, 24, 40, 129), (2, 2, 10, 6, 70), (1, 1, 128, 64, 257), (2, 2, 128, 128, 511),
                                       (2, 2, 72, 8, 256), (1, 1, 136, 16, 90), (4, 2, 64, 64, 1)])
def test_prompt_attention(device, H, G, D, V, T):
    """Far keys that stand out, at tile borders, in whole prompts and for the last queries alone, with and without gates."""
    far = [(i, j) for i, j in ((T - 1, 0), (T - 2, 127), (T - 3, 128), (200, 63), (128, 127), (128, 0), (127, 126), (64, 15), (16, 16)) if 0 <= j <= i < T]
    q, k, v = peaked(T, H, D, V, far, D)
    k, v = k[:, :G], v[:, :G]
    for i, j in far:
        q[i] = k[j].repeat_interleave(H // G, 0) * 2.0
    gate = torch.randn(T, H, generator=torch.Generator().manual_seed(1)) * 2
    scale = 3.0 * D ** -0.5
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        if device == "cpu" and dt == torch.bfloat16:
            continue
        c = lambda t: t.reshape(T, -1).to(dt)
        flat = K.rows(T, H * D + H, dt, device)
        flat.copy_(torch.cat([c(q), c(gate)], 1))
        qq, gg, kk, vv = flat[:, :H * D], flat[:, H * D:], c(k).to(device), c(v).to(device)
        u = lambda t, *s: t.to(dt).double().reshape(T, *s)
        plain = torch.stack([O.attend(u(q, H, D)[:, h], u(k, G, D)[:, h // (H // G)], u(v, G, V)[:, h // (H // G)], scale) for h in range(H)], 1)
        want = O.head_gate(plain, u(gate, H))
        close(K.head_attn(qq, kk, vv, 1, T, T, H, G, D, V, scale, gg).view(T, H, V), want, tol)
        close(K.head_attn(qq, kk, vv, 1, T, T, H, G, D, V, scale).view(T, H, V), plain, tol)
        n = (T + 2) // 3
        close(K.head_attn(qq[-n:], kk, vv, 1, n, T, H, G, D, V, scale, gg[-n:]).view(n, H, V), want[-n:], tol)
        two = lambda t: torch.cat([t, t.flip(0)])            # another sequence beside it
        o = K.head_attn(two(qq).contiguous() if (H * D) % 8 else two(flat)[:, :H * D], two(kk), two(vv), 2, T, T, H, G, D, V, scale, two(gg)).view(2, T, H, V)
        close(o[0], want, tol)


def shuffled_pages(T, seed=1, extra=3):
    n = (T + PAGE - 1) // PAGE
    order = torch.randperm(n + extra, generator=torch.Generator().manual_seed(seed))[:n]
    return order, order[torch.arange(T) // PAGE] * PAGE + torch.arange(T) % PAGE, (n + extra) * PAGE


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("T,R,eps", [(90, 40, 1e-5), (37, 22, 1e-2), (9, 512, 1e-6), (50, 33, 1e-3), (5, 1, 0.1)])
def test_latent_rows(device, T, R, eps):
    g = torch.Generator().manual_seed(R)
    order, slots, n = shuffled_pages(T)
    slots[T // 2] = -1
    for dt, tol in ((torch.float32, 1e-6), (torch.bfloat16, 1e-2)):
        src = K.rows(T, 24 + R + 3, dt, device)
        src.copy_(torch.randn(T, 24 + R + 3, generator=g))
        c, w = src[:, 24:24 + R], torch.randn(R, generator=g).to(dt)
        pool = torch.zeros(n, (R + 7) // 8 * 8, dtype=dt, device=device)
        got = K.latent_append(c, w.to(device), eps, slots.to(device), pool)
        want = O.rms(c.cpu().double(), eps) * w.double()
        close(got, want, tol)
        keep = slots >= 0
        assert torch.equal(pool[slots[keep].to(device), :R].cpu(), got.cpu()[keep])
        rest = torch.ones(n, dtype=torch.bool)
        rest[slots[keep]] = False
        assert not pool[rest.to(device)].any() and not pool[:, R:].any()
        K.latent_append(c, w.to(device), eps, slots.to(device), pool, want_rows=False)
        back = K.gather_rows(pool, order.int().to(device), 3, T - 4)[:, :R]
        assert torch.equal(back.cpu()[keep[3:T - 1]], got.cpu()[3:T - 1][keep[3:T - 1]])


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("M,H,D,R,V", [(1, 3, 16, 40, 48), (9, 2, 10, 22, 14), (65, 16, 128, 512, 128), (130, 5, 24, 72, 33), (16, 1, 7, 5, 3), (33, 40, 24, 200, 40)])
def test_head_products(device, M, H, D, R, V):
    g = torch.Generator().manual_seed(M)
    r = lambda *s: torch.randn(*s, generator=g)
    W = (R + 7) // 8 * 8
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        if device == "cpu" and dt == torch.bfloat16:
            continue
        def put(t):
            o = K.padded_weight(*t.shape, dt, device)
            o.copy_(t)
            return o
        q, ukv, gate = put(r(M, H * D + 3)), put(r(H * (D + V), R) * D ** -0.5), put(r(M, H))
        k64 = ukv.cpu().double()
        got = K.head_linear(q[:, :H * D], ukv[:H * D], H, D, R, transposed=True)
        want = torch.einsum("mhd,hdr->mhr", q[:, :H * D].cpu().double().view(M, H, D), k64[:H * D].view(H, D, R))
        assert got.shape == (M, H * W) and not got.reshape(M, H, W)[..., R:].any()
        close(got.reshape(M, H, W)[..., :R], want, tol)
        u = torch.zeros(M, H, W)
        u[..., :R] = r(M, H, R)
        u = put(u.view(M, H * W))
        want = torch.einsum("mhr,hvr->mhv", u.cpu().double().view(M, H, W)[..., :R], k64[H * D:].view(H, V, R))
        close(K.head_linear(u, ukv[H * D:], H, R, V).reshape(M, H, V), want, tol)
        close(K.head_linear(u, ukv[H * D:], H, R, V, gate=gate).reshape(M, H, V), O.head_gate(want, gate.cpu().double()), tol)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,R", [(6, 40), (16, 64), (20, 72), (40, 512), (3, 22), (16, 200), (5, 520), (32, 256), (1, 128)])
def test_latent_decode(device, H, R):
    """Keys that stand out at page and tile borders and far away, pages in a shuffled order with others' rows between them,
    sequences of unequal length, several splits."""
    T, W = 330, (R + 7) // 8 * 8
    g = torch.Generator().manual_seed(R)
    order, slots, n = shuffled_pages(T)
    c = O.rms(torch.randn(T, R, generator=g), 1e-5)
    pairs = [(329, 0), (328, 63), (327, 64), (320, 15), (319, 16), (200, 127), (130, 128), (129, 129), (64, 0), (63, 63), (15, 14), (1, 0), (0, 0), (300, 191)]
    at = [i for i, _ in pairs]
    q = torch.stack([torch.stack([c[(j + h) % (i + 1)] for h in range(H)]) for i, j in pairs]) * 2
    scale = 8.0 / R if R >= 8 else 1.0
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        if device == "cpu" and dt == torch.bfloat16:
            continue
        pool = torch.full((n, W), 9.0, dtype=dt, device=device)
        pool[:, R:] = 0
        pool[slots.to(device), :R] = c.to(dt).to(device)
        qq = torch.zeros(len(at), H, W, dtype=dt)
        qq[..., :R] = q.to(dt)
        cd, qd = c.to(dt).double(), qq[..., :R].double()
        want = torch.zeros(len(at), H, W, dtype=torch.float64)
        for b, i in enumerate(at):
            for h in range(H):
                want[b, h, :R] = O.attend_one(qd[b, h], cd[:i + 1], cd[:i + 1], scale)
        bt = order.int().to(device).repeat(len(at), 1)
        for splits in (None, 1, 3):
            got = K.latent_decode(qq.view(len(at), -1).to(device), pool, bt, torch.tensor(at, dtype=torch.int32, device=device), H, R, scale, splits=splits)
            close(got.reshape(len(at), H, W), want, tol)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("T,E,k", [(5, 6, 2), (300, 6, 2), (1, 1, 1), (64, 40, 5), (700, 300, 9), (3, 4, 4), (257, 3, 3), (256, 64, 6)])
def test_routing(device, T, E, k):
    """Large biases, equal logits, and rows: every assignment has one of its own, in a tile of its expert."""
    g = torch.Generator().manual_seed(T + E)
    z, b = torch.randn(T, E, generator=g), (torch.randn(E, generator=g) * 9).to(torch.bfloat16)
    z[T // 2] = -b.float()                            # all equal: the lower index first
    z[0] = z[0].round() - b.float()                   # ties
    r = X.route(z.to(device), b.to(device), k)
    for t in range(T):
        want = O.route((z[t] + b.float()).double(), k)
        assert r.idx[t].tolist() == [e for e, _ in want]
        assert max(abs(x - w) for x, (_, w) in zip(r.w[t].tolist(), want)) < 1e-5
    rows = r.row_of.reshape(-1).tolist()
    assert len(set(rows)) == T * k and max(rows) < r.max_rows == len(r.expert_of_tile) * 128
    tile = r.expert_of_tile.tolist()
    assert all(tile[x // 128] == e for x, e in zip(rows, r.idx.reshape(-1).tolist()))
    used = {x // 128 for x in rows}
    assert all((i in used) == (e >= 0) for i, e in enumerate(tile))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("T,H,E,k,F,Fs", [(5, 96, 6, 2, 24, 56), (70, 50, 3, 3, 7, 9), (300, 64, 9, 1, 33, 0), (1, 128, 40, 5, 96, 64), (400, 96, 4, 2, 40, 24)])
def test_mixture(device, T, H, E, k, F, Fs):
    c = TekenexConfig.from_dict(cfg(H, 11, [layer(1, 8, 8, 8, moe(E, k, F, Fs))]))
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        if device == "cpu" and dt == torch.bfloat16:
            continue
        m = TekenexModel(c, device=device, dtype=dt, seed=T)
        f = m.layers[0].mlp
        f.router_bias.data.copy_(torch.arange(E) * 0.7)
        h = K.rows(T, H, dt, device)
        h.copy_(torch.randn(T, H, generator=torch.Generator().manual_seed(T)))
        w = {n: t.cpu().double() for n, t in m.named_tensors()}
        p = "l0.mlp."
        three = lambda q: tuple(w[p + q + n] for n in (".gate", ".up", ".down"))
        hd = h.cpu().double()
        z = (hd @ w[p + "router"].T + w[p + "router.b"]).sort(-1, descending=True).values
        clear = torch.ones(T, dtype=torch.bool) if k == E else (z[:, k - 1] - z[:, k]) > 1e-3
        want = O.mixture(hd, w[p + "router"], w[p + "router.b"], k, [three(f"e{e}") for e in range(E)], three("shared") if Fs else None)
        got = f(h, lambda x, i, n, v, act=None: K.linear(x, v.data, act=act))
        assert int(clear.sum()) >= 0.9 * T
        close(got[clear.to(device)], want[clear], tol)
        if Fs:                                         # the shared expert is not a rounding
            less = O.mixture(hd, w[p + "router"], w[p + "router.b"], k, [three(f"e{e}") for e in range(E)])
            assert float((less - want).abs().max()) > 10 * tol


# ------------------------------------------------------------------------------------------------ the decoder
@pytest.mark.parametrize("run", RUNS, ids=str)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts(name, run):
    m, plain = build(name, *run)
    seq = toks(150, m.cfg.vocab_size)
    res, ref = [], []
    want = plain.run(seq, residuals=ref)
    got = m.head(m.hidden_states(torch.tensor([seq]), res))
    assert len(res) == len(ref)
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
    assert eng.cache.allocator.num_free == 64


@pytest.mark.parametrize("run", RUNS, ids=str)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_batches_of_unequal_requests(name, run):
    """Requests of unequal length prefilled and decoded together; some end early, their pages go to new requests, and every
    position equals the request alone."""
    m, plain = build(name, *run, seed=2)
    lens, V = [1, 70, 33, 17, 2], m.cfg.vocab_size
    seqs = [toks(l + 20, V, 10 + i) for i, l in enumerate(lens)]
    want = [plain.run(s) for s in seqs]
    eng = engine(m, max_batch=5, num_pages=24)
    for rep in range(2):                 # the second pass runs on pages the first one gave back
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
        assert eng.cache.allocator.num_free == 24


@pytest.mark.parametrize("run", RUNS, ids=str)
def test_long_decoding(run):
    m, plain = build("mixed", *run, seed=3)
    seq = toks(330, m.cfg.vocab_size, 3)
    want = plain.run(seq)
    assert off(feed_all(engine(m), seq, [20] + [1] * 310), want) < limit(run)


def test_faults_would_show():
    """The fp32 limit is far below what one wrong constant, a lost bias, scale, gate or shared expert does to these models' logits."""
    m, plain = build("mixed", seed=1)
    seq = toks(60, m.cfg.vocab_size, 1)
    want = plain.run(seq)
    far = 50 * limit(("cpu", "float32"))
    for change in (lambda c: c["layers"][1]["mixer"].update(scale=0.25), lambda c: c["norm"].update(eps=1e-2),
                   lambda c: c["layers"][0]["mlp"]["router"].update(top=1), lambda c: c["layers"][3]["mlp"]["router"].update(top=2),
                   lambda c: c["layers"][0]["mlp"].pop("shared")):
        other = json.loads(json.dumps(CONFIGS["mixed"]))
        change(other)
        assert off(O.PlainTekenex(other, plain.w).run(seq), want) > far
    for name, value in (("l0.ls1", 1.0), ("l2.norm1.b", 0.0), ("l1.mix.g", 0.0), ("l3.mlp.router.b", 0.0), ("l1.mix.dkv.norm", 1.0), ("final.norm.b", 0.0)):
        w = dict(plain.w, **{name: torch.full_like(plain.w[name], value)})
        assert off(O.PlainTekenex(CONFIGS["mixed"], w).run(seq), want) > far, name


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
    assert eng.generate_batch(prompts, 12, GREEDY) == want
    stop = want[1][3]
    r = eng.add_request(prompts[1], 12, GREEDY, stop_ids=(stop,))
    s = eng.add_request(prompts[0], 12, GREEDY)
    while eng.has_pending():
        eng.step()
    assert r.out == want[1][:want[1].index(stop) + 1] and s.out == want[0]
    assert eng.cache.allocator.num_free == 40


@pytest.mark.parametrize("run", RUNS[:2], ids=str)
def test_shared_prefixes(run):
    """Requests that share a prompt prefix reuse its pages of latents; the rest of the prompt attends over them."""
    m, plain = build("mixed", *run, seed=6)
    head = toks(50, 211, 1)
    prompts = [head + toks(n, 211, 40 + n) for n in (9, 1, 30)] + [head[:33]]
    eng = engine(m, enable_prefix_cache=True, max_batch=1)
    for p in prompts:
        assert eng.generate_batch([p], 6, GREEDY)[0] == plain.greedy(p, 6)
    assert eng.stats.prefix_hit_tokens == 48 + 48 + 32
    eng.prefix.evict_all()
    assert eng.cache.allocator.num_free == 64


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
    assert set(engine(m, weight_format="int8").packed) >= {"layers.0.proj", "layers.0.o", "layers.0.gate_up", "layers.1.up", "layers.1.down"}
    seq = toks(60, 300, 6)
    assert off(feed_all(engine(m, weight_format="int8"), seq, [40] + [1] * 20), plain.run(seq)) < 0.15


# ------------------------------------------------------------------------------------------------ configuration, folders, tools
def test_config_reader():
    for d in CONFIGS.values():
        c = TekenexConfig.from_dict(d)
        assert c.to_dict() == d
        m = TekenexModel(c, seed=None)
        assert m.param_count() == c.num_params() == sum(t.numel() for t in m.parameters())
        assert c.active_params() <= c.num_params()
    assert TekenexConfig.from_dict(CONFIGS["large"]).active_params() < TekenexConfig.from_dict(CONFIGS["large"]).num_params()
    for change, what in ((lambda l: l["mlp"]["router"].update(top=7), "choose 7 of 6"), (lambda l: l.update(type="attention"), "unknown mixer"),
                         (lambda l: l["mlp"].update(kind="other"), "unknown feed-forward"), (lambda l: l["mixer"].update(kv_rank=0), "positive")):
        bad = json.loads(json.dumps(CONFIGS["mixed"]))
        change(bad["layers"][0])
        with pytest.raises(ValueError, match=what):
            TekenexConfig.from_dict(bad)
    with pytest.raises(ValueError, match="kv_mode"):
        engine(TekenexModel(TekenexConfig.from_dict(CONFIGS["odd"])), kv_mode="fp8")


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    d = tmp_path_factory.mktemp("tekenex")
    m, plain = build("mixed", seed=7)
    registry.save_folder(m, d)
    return d, plain


def test_folder_roundtrip(folder):
    d, plain = folder
    m = registry.load_any(d)
    assert isinstance(m, TekenexModel) and m.lm_head is m.tok_embeddings
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
    assert "Architecture: Tekenex" in out and "layer 1: latent_attention heads=5 dim=32 vdim=8 kv_rank=24 ffn=160" in out
    assert "layer 0: latent_attention heads=3 dim=16 vdim=48 kv_rank=40 experts=6 top=2 ffn=24 shared=56" in out
    assert "tok/s]" in tool("quant_infer", d, "hi", "--max-tokens", 4, "--seed", 3)
