"""Plain, slow statements of the sequence mixers and of the decoder built from them, one function per mechanism, for the
tests to compare the framework with.  Everything is float64 NumPy-style torch on the CPU, one token or one head at a time
where that is clearest; nothing here is shared with the package."""
import math

import torch

DT = torch.float64


def silu(z):
    return z / (1 + torch.exp(-z))


def rms(x, eps):
    """x divided by the root of its mean square over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose stored weight is the deviation from one."""
    return rms(x, eps) * (1 + w)


def swiglu(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


# ---------------------------------------------------------------------------------------------------- rotation
def rope_angles(dims, base, scaling=None):
    """Frequencies [dims / 2] and the factor on cos and sin."""
    freqs = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            def where(turns):
                return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
            lo = max(math.floor(where(scaling["fast"])), 0)
            hi = min(math.ceil(where(scaling["slow"])), dims - 1)
            r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / scaling["factor"] * r + f * (1 - r)
        freqs.append(f)
    return freqs, (0.1 * math.log(scaling["factor"]) + 1.0) if scaling else 1.0


def rotate(x, pos, dims, base, scaling=None):
    """x [dim] at one position; the first ``dims`` entries are rotated, entry i with entry i + dims / 2."""
    freqs, m = rope_angles(dims, base, scaling)
    y = x.clone()
    for i, f in enumerate(freqs):
        c, s = math.cos(pos * f) * m, math.sin(pos * f) * m
        u, v = x[i], x[i + dims // 2]
        y[i] = u * c - v * s
        y[i + dims // 2] = v * c + u * s
    return y


def rotate_rows(x, pos0, dims, base, scaling=None):
    """The same for x [T, n, dim] at positions pos0, pos0 + 1, ..."""
    freqs, m = rope_angles(dims, base, scaling)
    a = torch.arange(pos0, pos0 + x.shape[0], dtype=DT)[:, None] * torch.tensor(freqs, dtype=DT)[None]
    c, s = (a.cos() * m)[:, None], (a.sin() * m)[:, None]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


# ---------------------------------------------------------------------------------------------------- attention
def visible(i, j, window=None):
    return j <= i and (window is None or i - j < window)


def attend_one(q, ks, vs, scale):
    """Softmax attention of one query over the given keys / values."""
    s = torch.stack([(q * k).sum() for k in ks]) * scale
    w = torch.exp(s - s.max())
    return (w[:, None] * torch.stack(list(vs))).sum(0) / w.sum()


def attend(q, k, v, scale, window=None):
    """q [T, dim] (the last T positions) over k [N, dim], v [N, vdim] with causality and an optional window."""
    T, N = q.shape[0], k.shape[0]
    i = torch.arange(N - T, N)[:, None]
    j = torch.arange(N)[None]
    ok = j <= i
    if window is not None:
        ok = ok & (i - j < window)
    s = (q @ k.T) * scale
    return torch.softmax(s.masked_fill(~ok, -math.inf), -1) @ v


def diff_lambda(lq1, lk1, lq2, lk2, diff):
    return float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff)


def diff_attend(q, k, v, heads, kv_heads, scale, lam, diff, eps, window=None):
    """Differential attention.  q [T, heads, 2, dim] and k [N, kv_heads, 2, dim] are rotated already, v [N, kv_heads, vdim];
    returns [T, heads, vdim]."""
    out = []
    for h in range(heads):
        g = h // (heads // kv_heads)
        a1 = attend(q[:, h, 0], k[:, g, 0], v[:, g], scale, window)
        a2 = attend(q[:, h, 1], k[:, g, 1], v[:, g], scale, window)
        out.append(rms(a1 - lam * a2, eps) * (1 - diff))
    return torch.stack(out, 1)


# ---------------------------------------------------------------------------------------------------- gated delta rule
def short_conv(x, w, past=None):
    """Causal convolution per channel: x [T, C], w [C, taps] (last column: the current token), ``past`` [taps - 1, C]
    inputs before x (zeros at the start).  Returns (silu of the result, the last taps - 1 inputs)."""
    taps = w.shape[1]
    past = torch.zeros(taps - 1, x.shape[1], dtype=x.dtype) if past is None else past
    full = torch.cat([past, x], 0)
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(taps):
            y[t] += w[:, j] * full[t + j]
    return silu(y), full[full.shape[0] - (taps - 1):]


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_scan(q, k, v, beta, g, state=None):
    """Gated delta rule of one head: q, k [T, dim] (unit length, q scaled), v [T, vdim], beta, g [T].  State [dim, vdim]."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=k.dtype) if state is None else state.clone()
    out = []
    for t in range(k.shape[0]):
        S = g[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out.append(S.T @ q[t])
    return torch.stack(out), S


# ---------------------------------------------------------------------------------------------------- the decoder
class PlainLanedra:
    """The whole decoder over a config dictionary and a dictionary of tensors; ``run`` takes the tokens of one sequence and
    returns logits, and can be called again with more tokens (``state`` carries keys, values and recurrent state)."""

    def __init__(self, cfg, tensors):
        self.cfg = cfg
        self.w = {n: t.to(DT) for n, t in tensors.items()}

    def start(self):
        return {"pos": 0, "layers": [{} for _ in self.cfg["layers"]]}

    def attention(self, i, h, st, pos):
        c, w, p = self.cfg["layers"][i]["mixer"], self.w, f"l{i}.mix."
        H, G, D, V = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
        T = h.shape[0]
        rot = (c["rot"]["dims"], c["rot"]["base"], c["rot"].get("scaling"))
        q = rotate_rows((h @ w[p + "q"].T).view(T, 2 * H, D), pos, *rot).view(T, H, 2, D)
        src = c.get("kv_from")
        if src is None:
            k = rotate_rows((h @ w[p + "k"].T).view(T, 2 * G, D), pos, *rot).view(T, G, 2, D)
            v = (h @ w[p + "v"].T).view(T, G, V)
            mine = st["layers"][i]
            mine["k"] = torch.cat([mine["k"], k]) if "k" in mine else k
            mine["v"] = torch.cat([mine["v"], v]) if "v" in mine else v
        else:
            mine = st["layers"][src]
        lam = diff_lambda(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], c["diff"])
        o = diff_attend(q, mine["k"], mine["v"], H, G, c["scale"], lam, c["diff"], self.cfg["norm"]["eps"],
                        c["mask"]["size"] if c.get("mask") else None)
        return o.reshape(T, H * V) @ w[p + "o"].T

    def delta(self, i, h, st):
        c, w, p = self.cfg["layers"][i]["mixer"], self.w, f"l{i}.mix."
        H, G, D, V = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
        T, mine = h.shape[0], st["layers"][i]
        x = {}
        for n in "qkv":
            x[n], mine["conv_" + n] = short_conv(h @ w[p + n].T, w[p + n + ".conv"], mine.get("conv_" + n))
        q = unit(x["q"].view(T, G, D)) * D ** -0.5
        k = unit(x["k"].view(T, G, D))
        v = x["v"].view(T, H, V)
        beta = 1 / (1 + torch.exp(-(h @ w[p + "b"].T)))
        z = h @ w[p + "a"].T + w[p + "dt_bias"]
        g = torch.exp(-torch.exp(w[p + "A_log"]) * torch.log1p(torch.exp(z)))
        outs, states = [], []
        for hd in range(H):
            gr = hd // (H // G)
            o, S = delta_scan(q[:, gr], k[:, gr], v[:, hd], beta[:, hd], g[:, hd], mine["S"][hd] if "S" in mine else None)
            outs.append(o)
            states.append(S)
        mine["S"] = states
        o = rms(torch.stack(outs, 1), self.cfg["norm"]["eps"]) * w[p + "norm"] * silu(h @ w[p + "g"].T).view(T, H, V)
        return o.reshape(T, H * V) @ w[p + "o"].T

    def run(self, tokens, st=None, residuals=None):
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        st = st if st is not None else self.start()
        x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
        for i, layer in enumerate(cfg["layers"]):
            p = f"l{i}."
            h = centred_norm(x, w[p + "norm1"], eps)
            y = self.attention(i, h, st, st["pos"]) if layer["type"] == "attention" else self.delta(i, h, st)
            x = x + centred_norm(y, w[p + "norm1b"], eps)
            if layer["mlp"] is not None:
                h = centred_norm(x, w[p + "norm2"], eps)
                y = swiglu(h, w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"])
                x = x + centred_norm(y, w[p + "norm2b"], eps)
            if residuals is not None:
                residuals.append(x.clone())
        st["pos"] += len(tokens)
        return centred_norm(x, w["final.norm"], eps) @ w["head"].T

    def greedy(self, tokens, n):
        st, out = self.start(), []
        lg = self.run(tokens, st)
        for _ in range(n):
            out.append(int(lg[-1].argmax()))
            lg = self.run([out[-1]], st)
        return out


# ---------------------------------------------------------------------------------------------------- latent attention
def layer_norm(x, w, b, eps):
    m = x.mean(-1, keepdim=True)
    d = x - m
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def latent_rows(h, dkv, norm, eps):
    """What latent attention remembers of a token: a projection of its input, divided by its root mean square and weighted."""
    return rms(h @ dkv.T, eps) * norm


def latent_attend(q, c, uk, uv, heads, dim, vdim, scale):
    """Softmax attention of q [T, heads * dim] (the last T positions) whose keys and values are read out of the latents c [N, rank],
    head by head; returns [T, heads, vdim]."""
    out = []
    for h in range(heads):
        k = c @ uk[h * dim:(h + 1) * dim].T
        v = c @ uv[h * vdim:(h + 1) * vdim].T
        out.append(attend(q[:, h * dim:(h + 1) * dim], k, v, scale))
    return torch.stack(out, 1)


def head_gate(o, z):
    """o [T, heads, vdim], one gate logit per head z [T, heads]."""
    return o / (1 + torch.exp(-z))[..., None]


# ---------------------------------------------------------------------------------------------------- feed-forwards
def relu2(z):
    return torch.where(z > 0, z * z, torch.zeros_like(z))


def squared_mlp(h, up, down):
    return relu2(h @ up.T) @ down.T


def route(z, top):
    """One token's router logits -> [(expert, weight)]: the ``top`` largest logits, softmax over those alone."""
    order = sorted(range(len(z)), key=lambda e: (-float(z[e]), e))[:top]
    e = [math.exp(float(z[i]) - float(z[order[0]])) for i in order]
    return [(i, x / sum(e)) for i, x in zip(order, e)]


def mixture(h, router, bias, top, experts, shared=None):
    """Gated feed-forward experts ((gate, up, down) each) chosen per token, plus one that every token runs."""
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for i, w in route(router @ h[t] + bias, top):
            out[t] += w * swiglu(h[t], *experts[i])
    return out if shared is None else out + swiglu(h, *shared)


class PlainTekenex:
    """As PlainLanedra, for layers of latent attention with dense or mixture feed-forwards, a layer norm and a scale on every
    sublayer's output and the embedding as the head."""

    def __init__(self, cfg, tensors):
        self.cfg = cfg
        self.w = {n: t.to(DT) for n, t in tensors.items()}

    def start(self):
        return {"pos": 0, "c": [torch.zeros(0, l["mixer"]["kv_rank"], dtype=DT) for l in self.cfg["layers"]]}

    def mixer(self, i, x, st):
        m, w, p = self.cfg["layers"][i]["mixer"], self.w, f"l{i}.mix."
        st["c"][i] = torch.cat([st["c"][i], latent_rows(x, w[p + "dkv"], w[p + "dkv.norm"], self.cfg["norm"]["eps"])])
        o = latent_attend(x @ w[p + "q"].T, st["c"][i], w[p + "uk"], w[p + "uv"], m["heads"], m["dim"], m["vdim"], m["scale"])
        return head_gate(o, x @ w[p + "g"].T).reshape(x.shape[0], -1) @ w[p + "o"].T

    def ff(self, i, x):
        m, w, p = self.cfg["layers"][i]["mlp"], self.w, f"l{i}.mlp."
        if m["kind"] == "dense":
            return squared_mlp(x, w[p + "up"], w[p + "down"])
        three = lambda q: tuple(w[p + q + n] for n in (".gate", ".up", ".down"))
        r = m["router"]
        return mixture(x, w[p + "router"], w[p + "router.b"], r["top"], [three(f"e{e}") for e in range(r["experts"])],
                       three("shared") if m.get("shared") else None)

    def norm(self, name, x):
        return layer_norm(x, self.w[name], self.w[name + ".b"], self.cfg["norm"]["eps"])

    def run(self, tokens, st=None, residuals=None):
        w = self.w
        st = st if st is not None else self.start()
        x = w["embed"][torch.tensor(tokens)]
        for i, layer in enumerate(self.cfg["layers"]):
            p = f"l{i}."
            x = x + self.norm(p + "norm1", self.mixer(i, x, st)) * w[p + "ls1"]
            if layer["mlp"] is not None:
                x = x + self.norm(p + "norm2", self.ff(i, x)) * w[p + "ls2"]
            if residuals is not None:
                residuals.append(x.clone())
        st["pos"] += len(tokens)
        return self.norm("final.norm", x) @ w["embed"].T

    greedy = PlainLanedra.greedy


# ---------------------------------------------------------------------------------------------------- attention with options
def plain_norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def rotate_linear(x, pos0, dims, base, factor=1.0):
    """x [T, n, dim] at positions pos0, pos0 + 1, ...: entry i of the first ``dims`` with entry i + dims / 2, all frequencies divided
    by ``factor``."""
    f = torch.tensor([float(base) ** (-2.0 * i / dims) / factor for i in range(dims // 2)], dtype=DT)
    a = (torch.arange(pos0, pos0 + x.shape[0], dtype=DT)[:, None] * f)[:, None]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin(), x[..., dims:]], -1)


def query_temperature(p, coef, every):
    """Factor of the query at position p."""
    return 1 + coef * math.log((p + 1) // every + 1)


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def seen(i, j, window=None, keep_first=0):
    """Whether position i looks at position j."""
    return (j <= i) & ((j < keep_first) | (True if window is None else i - j < window))


def attend_options(q, k, v, pos0, scale, window=None, keep_first=0, cap=None, sink=False, temp=None):
    """One head.  q [T, dim] at positions pos0 ..., k [N, dim] and v [N, vdim] at 0 ...; ``cap``: soft cap of the scores; ``sink``: one
    more key of score 0 that has no value; ``temp``: (coef, every) of the queries' factor."""
    at = range(pos0, pos0 + q.shape[0])
    ok = seen(torch.tensor(at)[:, None], torch.arange(k.shape[0])[None], window, keep_first)
    f = torch.tensor([query_temperature(p, *temp) if temp else 1.0 for p in at], dtype=DT)
    s = (q * f[:, None]) @ k.T * scale
    if cap:
        s = soft_cap(s, cap)
    m = torch.where(ok, s, -math.inf).max(-1, keepdim=True).values.clamp(min=0)
    e = torch.where(ok, torch.exp(s - m), 0.0)
    return (e @ v) / (e.sum(-1, keepdim=True) + (torch.exp(-m) if sink else 0.0))


# ---------------------------------------------------------------------------------------------------- gated linear attention
def channel_decay(z, tau):
    return sigmoid(z) ** (1 / tau)


def gated_linear_scan(q, k, v, alpha, state=None):
    """One head: q, k, alpha [T, dim], v [T, vdim]; the state [dim, vdim] decays by key channel.  Returns (o [T, vdim], state)."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=k.dtype) if state is None else state.clone()
    out = []
    for t in range(k.shape[0]):
        S = alpha[t][:, None] * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out), S


# ---------------------------------------------------------------------------------------------------- feed-forwards
def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def geglu(h, gate, up, down):
    return (gelu_tanh(h @ gate.T) * (h @ up.T)) @ down.T


def route_groups(z, top, groups, keep, scale):
    """One token's router logits -> [(expert, weight)].  Scores are sigmoids; the ``keep`` groups of neighbouring experts with the
    largest sums of two scores stay; of their experts the ``top`` best, weighted by their scores over the scores' sum, times scale."""
    s = [1 / (1 + math.exp(-float(x))) for x in z]
    n = len(s) // groups
    mark = [sum(sorted(s[g * n:(g + 1) * n], reverse=True)[:2]) for g in range(groups)]
    stay = sorted(range(groups), key=lambda g: (-mark[g], g))[:keep]
    order = sorted((e for e in range(len(s)) if e // n in stay), key=lambda e: (-s[e], e))[:top]
    total = sum(s[e] for e in order) + 1e-20
    return [(e, s[e] / total * scale) for e in order]


def grouped_mixture(h, router, top, groups, keep, scale, experts, shared=None, shared_gate=None):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for i, w in route_groups(router @ h[t], top, groups, keep, scale):
            out[t] += w * swiglu(h[t], *experts[i])
    return out if shared is None else out + sigmoid(h @ shared_gate.T) * swiglu(h, *shared)


class PlainFigudra:
    """As PlainLanedra, for parallel layers (one norm, mixer and feed-forward side by side) of attention with options or gated linear
    attention, whose tensors may be those of another layer, under a normed embedding."""

    def __init__(self, cfg, tensors):
        self.cfg = cfg
        self.w = {n: t.to(DT) for n, t in tensors.items()}

    def start(self):
        return {"pos": 0, "layers": [{} for _ in self.cfg["layers"]]}

    def attention(self, m, p, h, mine, pos, eps):
        w, H, G, D, V, T = self.w, m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
        q, k, v = (h @ w[p + "q"].T).view(T, H, D), (h @ w[p + "k"].T).view(T, G, D), (h @ w[p + "v"].T).view(T, G, V)
        second = "rot" in m
        if second:
            rot = (m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling", {}).get("factor", 1.0))
            q = rotate_linear(plain_norm(q, w[p + "q.norm"], eps), pos, *rot)
            k = rotate_linear(plain_norm(k, w[p + "k.norm"], eps), pos, *rot)
            opt = dict(window=m["mask"]["size"], keep_first=m["mask"]["keep_first"], sink=True)
        else:
            opt = dict(cap=m["softcap"], temp=(m["q_temp"]["coef"], m["q_temp"]["every"]))
        mine["k"] = torch.cat([mine["k"], k]) if "k" in mine else k
        mine["v"] = torch.cat([mine["v"], v]) if "v" in mine else v
        o = torch.stack([attend_options(q[:, x], mine["k"][:, x // (H // G)], mine["v"][:, x // (H // G)], pos, m["scale"], **opt)
                         for x in range(H)], 1).reshape(T, H * V)
        if not second:
            o = o * sigmoid(h @ w[p + "g"].T)
        return o @ w[p + "o"].T

    def gla(self, m, p, h, mine, pos, eps):
        w, H, D, V, T = self.w, m["heads"], m["dim"], m["vdim"], h.shape[0]
        q, k, v = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5, (h @ w[p + "k"].T).view(T, H, D), (h @ w[p + "v"].T).view(T, H, V)
        a = channel_decay((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"], m["tau"]).view(T, H, D)
        both = [gated_linear_scan(q[:, x], k[:, x], v[:, x], a[:, x], mine["S"][x] if "S" in mine else None) for x in range(H)]
        mine["S"] = [s for _, s in both]
        o = plain_norm(torch.stack([o for o, _ in both], 1), w[p + "norm"], eps) * silu(h @ w[p + "g"].T).view(T, H, V)
        return o.reshape(T, H * V) @ w[p + "o"].T

    def ff(self, m, p, h):
        three = lambda q: tuple(self.w[p + q + n] for n in ("gate", "up", "down"))
        if m["kind"] == "dense":
            return geglu(h, *three(""))
        r = m["router"]
        return grouped_mixture(h, self.w[p + "router"], r["top"], r["groups"]["count"], r["groups"]["keep"], r["scale"],
                               [three(f"e{e}.") for e in range(r["experts"])], three("shared.") if m.get("shared") else None,
                               self.w.get(p + "shared.sg"))

    def run(self, tokens, st=None, residuals=None):
        w, eps = self.w, self.cfg["norm"]["eps"]
        st = st if st is not None else self.start()
        x = plain_norm(w["embed"][torch.tensor(tokens)], w["embed.norm"], eps)
        for i, l in enumerate(self.cfg["layers"]):
            p = f"l{l.get('weights_of', i)}."
            h = plain_norm(x, w[p + "norm1"], eps)
            y = (self.gla if l["type"] == "gla" else self.attention)(l["mixer"], p + "mix.", h, st["layers"][i], st["pos"], eps)
            x = x + (y + self.ff(l["mlp"], p + "mlp.", h) if l["mlp"] else y)
            if residuals is not None:
                residuals.append(x.clone())
        st["pos"] += len(tokens)
        return plain_norm(x, w["final.norm"], eps) @ w["head"].T

    greedy = PlainLanedra.greedy


# ---------------------------------------------------------------------------------------------------- chunked attention
def seen_in_chunk(i, j, size):
    """Whether position i looks at position j: earlier or the same, in the same chunk of ``size`` positions."""
    return (j <= i) & (i // size == j // size)


def attend_chunk(q, k, v, pos0, scale, size, sink=None, temp=1.0):
    """One head.  q [T, dim] at positions pos0 ..., k [N, dim] and v [N, vdim] at 0 ...; ``sink``: a number whose exponential joins the
    denominator; ``temp``: a factor of the scores."""
    at = torch.arange(pos0, pos0 + q.shape[0])
    ok = seen_in_chunk(at[:, None], torch.arange(k.shape[0])[None], size)
    s = torch.where(ok, q @ k.T * scale * temp, -math.inf)
    m = s.max(-1, keepdim=True).values
    if sink is not None:
        m = m.clamp(min=float(sink))
    e = torch.exp(s - m)
    return (e @ v) / (e.sum(-1, keepdim=True) + (torch.exp(sink - m) if sink is not None else 0.0))


# ---------------------------------------------------------------------------------------------------- recurrences over a matrix state
def forget_gate(z, lower):
    """Between ``lower`` and one."""
    return lower + (1 - lower) * sigmoid(z)


def hgrn2_scan(q, f, v, state=None):
    """One head: what is not kept is written, with no key of its own.  q, f [T, dim], v [T, vdim]."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(q.shape[0]):
        S = torch.diag(f[t]) @ S + torch.outer(1 - f[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out), S


def retention_scan(q, k, v, decay, state=None):
    """One head with one decay.  q, k [T, dim] (rotated, k scaled), v [T, vdim]."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(q.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out), S


# ---------------------------------------------------------------------------------------------------- grouped norm, streams
def group_norm(x, w, groups, eps):
    """RMS norm of every one of ``groups`` equal consecutive parts; one weight for the whole."""
    return torch.cat([rms(p, eps) for p in x.chunk(groups, -1)], -1) * w


def streams_in(xs, coef):
    """What a sublayer reads of the streams xs (a list)."""
    return sum(float(c) * x for c, x in zip(coef, xs))


def streams_out(xs, y, mix, out):
    """The streams behind a sublayer that returned y; mix [from, to]."""
    return [sum(float(mix[s, t]) * xs[s] for s in range(len(xs))) + float(out[t]) * y for t in range(len(xs))]


# ---------------------------------------------------------------------------------------------------- clamped experts
def clamped_glu(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ down.T


def route_all(z, top):
    """One token's router logits -> [(expert, weight)]: the softmax over all experts, of which the ``top`` largest keep their values."""
    m = max(float(x) for x in z)
    e = [math.exp(float(x) - m) for x in z]
    order = sorted(range(len(e)), key=lambda i: (-e[i], i))[:top]
    return [(i, e[i] / sum(e)) for i in order]


def clamped_mixture(h, router, top, experts, limit, shared=None, shared_limit=None):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for i, w in route_all(router @ h[t], top):
            out[t] += w * clamped_glu(h[t], *experts[i], limit)
    return out if shared is None else out + clamped_glu(h, *shared, shared_limit)


class PlainToderax:
    """As PlainLanedra, for hyper-connected layers of HGRN2 or of chunked attention and retention side by side."""

    def __init__(self, cfg, tensors):
        self.cfg = cfg
        self.w = {n: t.to(DT) for n, t in tensors.items()}

    def start(self):
        return {"pos": 0, "layers": [{} for _ in self.cfg["layers"]]}

    def hgrn2(self, m, p, h, mine, pos, eps):
        w, H, D, V, T = self.w, m["heads"], m["dim"], m["vdim"], h.shape[0]
        q, v = silu(h @ w[p + "q"].T).view(T, H, D), (h @ w[p + "v"].T).view(T, H, V)
        f = forget_gate(h @ w[p + "f"].T + w[p + "f.b"], w[p + "lower"]).view(T, H, D)
        both = [hgrn2_scan(q[:, x], f[:, x], v[:, x], mine["S"][x] if "S" in mine else None) for x in range(H)]
        mine["S"] = [s for _, s in both]
        return plain_norm(torch.stack([o for o, _ in both], 1), w[p + "norm"], eps).reshape(T, H * V) @ w[p + "o"].T

    def chunked(self, m, p, h, mine, pos, eps):
        w, H, G, D, V, T = self.w, m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
        q, k, v = ((h @ w[p + n].T + w[p + n + ".b"]).view(T, c, -1) for n, c in (("q", H), ("k", G), ("v", G)))
        q, k = rms(q, eps), rms(k, eps)
        mine["k"] = torch.cat([mine["k"], k]) if "k" in mine else k
        mine["v"] = torch.cat([mine["v"], v]) if "v" in mine else v
        o = torch.stack([attend_chunk(q[:, x], mine["k"][:, x // (H // G)], mine["v"][:, x // (H // G)], pos, m["scale"], m["mask"]["size"],
                                      w[p + "sink"][x], w[p + "temp"][x]) for x in range(H)], 1)
        return o.reshape(T, H * V) @ w[p + "o"].T

    def retention(self, m, p, h, mine, pos, eps):
        w, H, D, V, T = self.w, m["heads"], m["dim"], m["vdim"], h.shape[0]
        turn = lambda x: rotate_linear(x.view(T, H, D), pos, m["rot"]["dims"], m["rot"]["base"])
        q, k, v = turn(h @ w[p + "q"].T), turn(h @ w[p + "k"].T) * D ** -0.5, (h @ w[p + "v"].T).view(T, H, V)
        both = [retention_scan(q[:, x], k[:, x], v[:, x], m["decay"][x], mine["S"][x] if "S" in mine else None) for x in range(H)]
        mine["S"] = [s for _, s in both]
        o = rms(torch.stack([o for o, _ in both], 1), eps).reshape(T, H * V)
        return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T

    def mixer(self, l, p, h, mine, pos, eps):
        if l["type"] == "hgrn2":
            return self.hgrn2(l["mixer"], p, h, mine, pos, eps)
        a = self.chunked(l["mixer"]["left"], p + "left.", h, mine.setdefault("left", {}), pos, eps)
        b = self.retention(l["mixer"]["right"], p + "right.", h, mine.setdefault("right", {}), pos, eps)
        return (plain_norm(a, self.w[p + "left.out"], eps) + plain_norm(b, self.w[p + "right.out"], eps)) / 2

    def ff(self, m, p, h):
        three = lambda q: tuple(self.w[p + q + n] for n in (".gate", ".up", ".down"))
        r, s = m["router"], m.get("shared")
        return clamped_mixture(h, self.w[p + "router"], r["top"], [three(f"e{e}") for e in range(r["experts"])], m["expert"]["limit"],
                               three("shared") if s else None, s["limit"] if s else None)

    def run(self, tokens, st=None, residuals=None):
        c, w = self.cfg, self.w
        eps, groups = c["norm"]["eps"], c["norm"]["groups"]
        st = st if st is not None else self.start()
        xs = [w["embed"][torch.tensor(tokens)] * c["embedding"]["scale"]] * c["streams"]
        for i, l in enumerate(c["layers"]):
            p = f"l{i}."
            for n, sub in ((1, lambda h: self.mixer(l, p + "mix.", h, st["layers"][i], st["pos"], eps)), (2, lambda h: self.ff(l["mlp"], p + "mlp.", h))):
                if n == 2 and l["mlp"] is None:
                    continue
                y = sub(group_norm(streams_in(xs, w[f"{p}hc{n}.in"]), w[f"{p}norm{n}"], groups, eps))
                xs = streams_out(xs, y, w[f"{p}hc{n}.mix"], w[f"{p}hc{n}.out"])
            if residuals is not None:
                residuals.append(sum(xs))
        st["pos"] += len(tokens)
        return group_norm(sum(xs), w["final.norm"], groups, eps) @ w["head"].T

    greedy = PlainLanedra.greedy
