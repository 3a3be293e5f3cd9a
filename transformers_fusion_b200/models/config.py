"""Model configuration.

``TransformerConfig`` mirrors the reference struct field for field
(include/quant/transformer.h:12-43) and serialises to the same raw 128-byte little-endian image
the reference writes into the ``.quant`` header (src/model/model.cpp:219-220), so checkpoints are
interchangeable.  Byte offsets (x86-64): vocab_size@0 i64, hidden_size@8, num_layers@16,
num_heads@24, head_dim@32, ffn_hidden_size@40, norm_eps@48 f32, rope_theta@52 f32, max_seq_len@56
i64, activation@64 u8, num_kv_heads@72 i64, use_parallel_residual@80 bool, mtp_num_heads@84 i32,
mtp_loss_weight@88 f32, rope_scaling_mode@92 u8, rope_scaling_factor@96 f32,
rope_original_max_seq_len@104 i64, yarn_attn_factor@112 f32, yarn_beta_fast@116 f32,
yarn_beta_slow@120 f32, use_fp8@124 bool, fp8_use_e4m3@125 bool.
"""
from __future__ import annotations

import struct
from dataclasses import asdict, dataclass, field

ACTIVATIONS = ["none", "relu", "gelu", "silu", "swiglu", "geglu"]
ROPE_SCALING = ["none", "linear", "ntk", "yarn"]
CONFIG_BYTES = 128


@dataclass
class TransformerConfig:
    vocab_size: int = 32000
    hidden_size: int = 512
    num_layers: int = 8
    num_heads: int = 8
    head_dim: int = 0            # 0 -> hidden_size // num_heads
    ffn_hidden_size: int = 0     # 0 -> 4 * hidden_size
    norm_eps: float = 1e-5
    rope_theta: float = 10000.0
    max_seq_len: int = 2048
    activation: str = "swiglu"
    num_kv_heads: int = 0        # 0 -> num_heads
    use_parallel_residual: bool = False
    mtp_num_heads: int = 0
    mtp_loss_weight: float = 0.0
    rope_scaling_mode: str = "none"
    rope_scaling_factor: float = 1.0
    rope_original_max_seq_len: int = 0
    yarn_attn_factor: float = 1.0
    yarn_beta_fast: float = 32.0
    yarn_beta_slow: float = 1.0
    use_fp8: bool = False
    fp8_use_e4m3: bool = True
    # ---- not part of the 128-byte image (kept in the JSON side-car / constructor only) ----
    tie_embeddings: bool = False
    norm_type: str = "rmsnorm"   # "layernorm" for the GPT-2-shaped variant
    position_type: str = "rope"  # "learned" for the GPT-2-shaped variant
    attention_bias: bool = False
    init_std: float = 0.02

    def __post_init__(self):
        if not self.head_dim:
            self.head_dim = self.hidden_size // self.num_heads
        if not self.ffn_hidden_size:
            self.ffn_hidden_size = 4 * self.hidden_size
        if not self.num_kv_heads:
            self.num_kv_heads = self.num_heads
        assert self.num_heads % self.num_kv_heads == 0
        self.activation = self.activation.lower()
        assert self.activation in ACTIVATIONS

    @property
    def gated(self) -> bool:
        return self.activation in ("swiglu", "geglu")

    @property
    def act_kernel(self) -> str:
        return {"swiglu": "silu", "geglu": "gelu"}.get(self.activation, self.activation)

    def num_params(self) -> int:
        H, F, D = self.hidden_size, self.ffn_hidden_size, self.head_dim
        per_layer = H * (self.num_heads + 2 * self.num_kv_heads) * D + self.num_heads * D * H
        per_layer += (3 if self.gated else 2) * H * F + 2 * H
        n = self.num_layers * per_layer + self.vocab_size * H + H
        if not self.tie_embeddings:
            n += self.vocab_size * H
        return n

    def flops_per_token(self, seq_len: int, causal: bool = True) -> float:
        """Training FLOPs per token (forward + backward = 3x forward matmul FLOPs)."""
        H, F, D = self.hidden_size, self.ffn_hidden_size, self.head_dim
        lin = H * (self.num_heads + 2 * self.num_kv_heads) * D + self.num_heads * D * H
        lin += (3 if self.gated else 2) * H * F
        attn = 2 * self.num_heads * D * seq_len * (0.5 if causal else 1.0)
        return 6.0 * (self.num_layers * (lin + attn) + self.vocab_size * H)

    # ------------------------------------------------------------------ binary image
    def to_bytes(self) -> bytes:
        b = bytearray(CONFIG_BYTES)
        struct.pack_into("<6q", b, 0, self.vocab_size, self.hidden_size, self.num_layers, self.num_heads,
                         self.head_dim, self.ffn_hidden_size)
        struct.pack_into("<ffq", b, 48, self.norm_eps, self.rope_theta, self.max_seq_len)
        b[64] = ACTIVATIONS.index(self.activation)
        struct.pack_into("<q", b, 72, self.num_kv_heads)
        b[80] = int(self.use_parallel_residual)
        struct.pack_into("<if", b, 84, self.mtp_num_heads, self.mtp_loss_weight)
        b[92] = ROPE_SCALING.index(self.rope_scaling_mode)
        struct.pack_into("<f", b, 96, self.rope_scaling_factor)
        struct.pack_into("<q", b, 104, self.rope_original_max_seq_len)
        struct.pack_into("<fff", b, 112, self.yarn_attn_factor, self.yarn_beta_fast, self.yarn_beta_slow)
        b[124] = int(self.use_fp8)
        b[125] = int(self.fp8_use_e4m3)
        return bytes(b)

    @classmethod
    def from_bytes(cls, raw: bytes, **extra) -> "TransformerConfig":
        if len(raw) < CONFIG_BYTES:
            raw = raw + bytes(CONFIG_BYTES - len(raw))
        v, h, nl, nh, hd, ff = struct.unpack_from("<6q", raw, 0)
        eps, theta, msl = struct.unpack_from("<ffq", raw, 48)
        (nkv,) = struct.unpack_from("<q", raw, 72)
        mtp_n, mtp_w = struct.unpack_from("<if", raw, 84)
        (rsf,) = struct.unpack_from("<f", raw, 96)
        (romsl,) = struct.unpack_from("<q", raw, 104)
        yaf, ybf, ybs = struct.unpack_from("<fff", raw, 112)
        act = raw[64] if raw[64] < len(ACTIVATIONS) else 0
        rsm = raw[92] if raw[92] < len(ROPE_SCALING) else 0
        return cls(vocab_size=v, hidden_size=h, num_layers=nl, num_heads=nh, head_dim=hd, ffn_hidden_size=ff,
                   norm_eps=eps, rope_theta=theta, max_seq_len=msl, activation=ACTIVATIONS[act], num_kv_heads=nkv,
                   use_parallel_residual=bool(raw[80]), mtp_num_heads=mtp_n, mtp_loss_weight=mtp_w,
                   rope_scaling_mode=ROPE_SCALING[rsm], rope_scaling_factor=rsf or 1.0,
                   rope_original_max_seq_len=romsl, yarn_attn_factor=yaf or 1.0, yarn_beta_fast=ybf or 32.0,
                   yarn_beta_slow=ybs or 1.0, use_fp8=bool(raw[124]), fp8_use_e4m3=bool(raw[125]), **extra)

    def to_dict(self):
        return asdict(self)


@dataclass
class MoEConfig(TransformerConfig):
    """Sparse mixture-of-experts decoder (reference: include/quant/moe_model.h, moe_variants.h:61-123)."""
    num_experts: int = 8
    top_k: int = 2
    expert_hidden_size: int = 0          # 0 -> ffn_hidden_size
    num_shared_experts: int = 0
    load_balance_weight: float = 0.01
    router_z_weight: float = 0.001
    capacity_factor: float = 2.0
    capacity_policy: str = "none"        # none | fixed | token_drop | token_pass
    renormalize_topk: bool = True        # softmax over the selected k (Mixtral); False = reference SparseMoE
    variant: str = "sparse_topk"
    expert_fp8: bool = False             # block-scaled E4M3 expert GEMMs

    def __post_init__(self):
        super().__post_init__()
        if not self.expert_hidden_size:
            self.expert_hidden_size = self.ffn_hidden_size


# ---------------------------------------------------------------------------------------------------------------------
# decoders described layer by layer: every layer names its sequence mixer and its feed-forward
# ---------------------------------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class RotarySpec:
    """Rotary embedding of the first ``dims`` entries of a head; ``yarn_*`` (factor None: unscaled) as in YaRN; ``linear``: every
    frequency is divided by it."""
    dims: int
    base: float
    yarn_factor: float = None
    yarn_original: int = 0
    yarn_fast: float = 32.0
    yarn_slow: float = 1.0
    linear: float = 1.0


def first_key(pos: int, window: int = 0, chunk: int = 0) -> int:
    """The first position that a query at ``pos`` looks at: of its window, or of its chunk of positions, or 0."""
    return max(0, pos - window + 1) if window else pos // chunk * chunk if chunk else 0


@dataclass(frozen=True)
class DiffAttentionSpec:
    """Differential attention: per head two query / key maps of ``dim`` entries over one set of values of ``vdim`` entries.
    ``window`` 0: plain causal.  ``kv_from``: index of the layer whose keys and values this layer uses instead of its own."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot: RotarySpec
    window: int = 0
    kv_from: int = None

    kind = "attention"


@dataclass(frozen=True)
class GatedDeltaSpec:
    """Gated delta rule: ``kv_heads`` query / key heads of ``dim`` entries, ``heads`` value heads of ``vdim`` entries with a
    [dim, vdim] state each, after a causal convolution of ``conv`` taps on q, k and v."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    kind = "delta"

    @property
    def conv_channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Latent attention without positions: the keys (``dim`` entries) and values (``vdim``) of every head are read out of one
    latent of ``kv_rank`` entries per token, which is all that is cached; one output gate per head."""
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float

    kind = "latent_attention"
    window = 0

    @property
    def latent_width(self) -> int:
        """Entries of a cached row: the latent, padded to 16 bytes in bf16."""
        return (self.kv_rank + 7) // 8 * 8


@dataclass(frozen=True)
class HeadAttentionSpec:
    """Softmax attention of ``heads`` query heads over ``kv_heads`` key / value heads.  ``rot``: rotation of queries and keys (None:
    no positions); ``qk_norm``: RMS norm of every query and key head in front of it; ``gate``: one output gate per entry of the
    heads; ``window`` > 0: a position sees that many keys up to itself, and the first ``keep_first`` of the sequence; ``softcap``
    > 0: scores are cap tanh(score / cap); ``sink``: the denominator counts one more key of score 0; queries at position p are
    multiplied by 1 + temp_coef ln(floor((p + 1) / temp_every) + 1).  ``chunk`` > 0 (instead of a window): a position sees its own chunk of
    so many positions; ``bias``: on the projections of q, k and v; ``qk_weight``: the norms have a learnt weight; ``head_temp``: a learnt
    factor of the scores per head (with ``qk_norm``); ``head_sink``: a learnt score of the sink per head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotarySpec = None
    qk_norm: bool = False
    gate: bool = False
    window: int = 0
    keep_first: int = 0
    softcap: float = 0.0
    sink: bool = False
    temp_coef: float = 0.0
    temp_every: int = 1
    chunk: int = 0
    bias: bool = False
    qk_weight: bool = True
    head_temp: bool = False
    head_sink: bool = False

    kind = "head_attention"

    def params(self, hidden: int) -> int:
        q, kv, o = self.heads * self.dim, self.kv_heads * (self.dim + self.vdim), self.heads * self.vdim
        return hidden * (q + kv + o * (2 if self.gate else 1)) + (q + kv if self.bias else 0) + \
            (2 * self.dim if self.qk_norm and self.qk_weight else 0) + self.heads * (int(self.head_temp) + int(self.head_sink))


@dataclass(frozen=True)
class GatedLinearSpec:
    """Gated linear attention: per head a [dim, vdim] state whose rows decay by sigmoid(z)^(1/tau), z from a projection of rank
    ``rank`` per key channel."""
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int = 16

    kind = "gla"


@dataclass(frozen=True)
class ForgetLinearSpec:
    """Linear attention whose forget gate also decides what is written (HGRN2): per head a [dim, vdim] state whose rows keep a share of
    themselves, at least a lower bound per channel, and take the rest from the values."""
    heads: int
    dim: int
    vdim: int

    kind = "hgrn2"

    def params(self, hidden: int) -> int:
        return hidden * self.heads * 2 * (self.dim + self.vdim) + 2 * self.heads * self.dim + self.vdim


@dataclass(frozen=True)
class RetentionSpec:
    """Retention: linear attention with one fixed decay per head, rotated queries and keys, and a gate per entry of the heads."""
    heads: int
    dim: int
    vdim: int
    decay: tuple
    rot: RotarySpec = None

    kind = "retention"

    def params(self, hidden: int) -> int:
        return hidden * self.heads * (2 * self.dim + 3 * self.vdim)


@dataclass(frozen=True)
class PairSpec:
    """Two mixers side by side on the same input; the result is half the sum of their outputs, each normed."""
    left: object
    right: object

    kind = "pair"

    def params(self, hidden: int) -> int:
        return self.left.params(hidden) + self.right.params(hidden) + 2 * hidden


def mixers_of(m):
    """The mixers that a layer's mixer consists of."""
    return (m.left, m.right) if m.kind == "pair" else (m,)


@dataclass(frozen=True)
class MixtureSpec:
    """Mixture of gated feed-forward experts: ``top`` of ``experts`` per token; ``shared_ff`` > 0: one more expert of that size that
    every token runs (``shared_gate``: times the sigmoid of a logit per token).  ``score`` "softmax": the largest logits (plus a
    bias), weighted by the softmax over the chosen ones.  "sigmoid": the largest sigmoids (no bias) among the experts of the ``keep``
    best of ``groups`` equal groups (by the sum of a group's two largest), weighted by them over their sum, times ``scale``.
    "softmax_all": the largest of the softmax over all experts (no bias), weighted by themselves.  ``act``: the gated unit (``stack.glu``),
    with its ``limit`` and that of the shared expert."""
    experts: int
    top: int
    ff: int
    shared_ff: int = 0
    shared_gate: bool = False
    score: str = "softmax"
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    act: str = "silu"
    limit: float = 0.0
    shared_limit: float = 0.0


@dataclass(frozen=True)
class StackLayer:
    mixer: object
    ffn_hidden_size: int = 0     # dense feed-forward; 0: the layer has none
    mixture: MixtureSpec = None  # mixture of experts instead of a dense feed-forward
    weights_of: int = None       # the layer whose tensors this one uses


@dataclass
class LanedraConfig:
    """Lanedra: differential sliding-window attention (optionally on another layer's keys and values) and gated-delta-rule
    layers in any order, norms before and after every sublayer, a 32-bit residual stream, a scaled embedding and a separate
    output head.  ``from_dict`` reads the model folder's config.json; the folder sets no context limit, so ``max_seq_len``
    is what the serving tables are sized for unless the engine's configuration says otherwise."""
    vocab_size: int
    hidden_size: int
    layers: list
    norm_eps: float
    embedding_scale: float = 1.0
    max_seq_len: int = 32768

    architecture = "Lanedra"
    tie_embeddings = False

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            m = l.mixer
            if m.heads % m.kv_heads:
                raise ValueError(f"layer {i}: {m.heads} heads do not divide over {m.kv_heads} kv heads")
            if m.kind == "attention":
                if m.rot.dims % 2 or not 0 < m.rot.dims <= m.dim:
                    raise ValueError(f"layer {i}: cannot rotate {m.rot.dims} of {m.dim} entries")
                if m.kv_from is not None:
                    src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                    if src is None or src.kind != "attention" or src.kv_from is not None:
                        raise ValueError(f"layer {i}: layer {m.kv_from} has no keys and values to share")
                    if (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
                        raise ValueError(f"layer {i}: layer {m.kv_from}'s keys and values have other sizes")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def window(self) -> int:
        """Keys that any attention layer may still look at, the current one included; 0: all of them."""
        w = [l.mixer.window for l in self.layers if l.mixer.kind == "attention"]
        return 0 if not w or 0 in w else max(w)

    @classmethod
    def from_dict(cls, d: dict, **extra) -> "LanedraConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            m = e["mixer"]
            if e["type"] == "attention":
                r = m["rot"]
                y = r.get("scaling")
                rot = RotarySpec(int(r["dims"]), float(r["base"])) if not y else \
                    RotarySpec(int(r["dims"]), float(r["base"]), float(y["factor"]), y["original"], float(y["fast"]), float(y["slow"]))
                mix = DiffAttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), float(m["diff"]), rot,
                                        (m.get("mask") or {}).get("size") or 0, m.get("kv_from"))
            elif e["type"] == "delta":
                mix = GatedDeltaSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
            else:
                raise ValueError(f"layer {i}: unknown mixer '{e['type']}'")
            mlp = e.get("mlp")
            if mlp and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
            layers.append(StackLayer(mix, mlp["ff"] if mlp else 0))
        return cls(vocab_size=d["vocab"], hidden_size=d["width"], layers=layers, norm_eps=float(d["norm"]["eps"]),
                   embedding_scale=float(d["embedding"]["scale"]), **extra)

    def to_dict(self) -> dict:
        """The config.json form."""
        out = []
        for l in self.layers:
            m = l.mixer
            x = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim}
            if m.kind == "delta":
                x["conv"] = m.conv
            else:
                r = {"dims": m.rot.dims, "base": m.rot.base}
                if m.rot.yarn_factor is not None:
                    r["scaling"] = {"factor": m.rot.yarn_factor, "original": m.rot.yarn_original, "fast": m.rot.yarn_fast,
                                    "slow": m.rot.yarn_slow}
                x.update(scale=m.scale, diff=m.diff, rot=r)
                if m.window:
                    x["mask"] = {"size": m.window}
                if m.kv_from is not None:
                    x["kv_from"] = m.kv_from
            out.append({"type": m.kind, "mixer": x, "mlp": {"kind": "dense", "ff": l.ffn_hidden_size} if l.ffn_hidden_size else None})
        return {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale}, "layers": out,
                "norm": {"eps": self.norm_eps}, "vocab": self.vocab_size, "width": self.hidden_size}

    def num_params(self) -> int:
        H, n = self.hidden_size, 2 * self.vocab_size * self.hidden_size + self.hidden_size
        for l in self.layers:
            m = l.mixer
            if m.kind == "attention":
                own = 0 if m.kv_from is not None else m.kv_heads * (2 * m.dim + m.vdim)
                n += H * (2 * m.heads * m.dim + own + m.heads * m.vdim) + 4 * m.dim
            else:
                n += H * (m.conv_channels + 2 * m.heads * m.vdim + 2 * m.heads) + m.conv_channels * m.conv + 2 * m.heads + m.vdim
            n += 2 * H + (3 * H * l.ffn_hidden_size + 2 * H if l.ffn_hidden_size else 0)
        return n


@dataclass
class TekenexConfig:
    """Tekenex: latent attention and dense (squared-relu) or mixture-of-experts feed-forwards in any order, a layer norm and a
    learnt per-channel scale on every sublayer's output (the sublayers read the 32-bit residual itself), the embedding table as
    the head.  ``from_dict`` reads the model folder's config.json; ``max_seq_len`` as in ``LanedraConfig``."""
    vocab_size: int
    hidden_size: int
    layers: list
    norm_eps: float
    max_seq_len: int = 32768

    architecture = "Tekenex"
    embedding_scale = 1.0
    tie_embeddings = True
    window = 0                   # every attention layer looks at all earlier keys

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            m, x = l.mixer, l.mixture
            if min(m.heads, m.dim, m.vdim, m.kv_rank) < 1:
                raise ValueError(f"layer {i}: sizes of the mixer have to be positive")
            if x is not None and not 1 <= x.top <= x.experts:
                raise ValueError(f"layer {i}: cannot choose {x.top} of {x.experts} experts")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: dict, **extra) -> "TekenexConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer '{e['type']}'")
            m, f = e["mixer"], e.get("mlp")
            mix = LatentAttentionSpec(m["heads"], m["dim"], m["vdim"], m["kv_rank"], float(m["scale"]))
            kind = f.get("kind", "dense") if f else None
            if kind == "dense":
                layers.append(StackLayer(mix, f["ff"]))
            elif kind == "moe":
                r, sh = f["router"], f.get("shared")
                layers.append(StackLayer(mix, 0, MixtureSpec(r["experts"], r["top"], f["expert"]["ff"], sh["ff"] if sh else 0)))
            elif kind is None:
                layers.append(StackLayer(mix))
            else:
                raise ValueError(f"layer {i}: unknown feed-forward '{kind}'")
        return cls(vocab_size=d["vocab"], hidden_size=d["width"], layers=layers, norm_eps=float(d["norm"]["eps"]), **extra)

    def to_dict(self) -> dict:
        """The config.json form."""
        out = []
        for l in self.layers:
            m, x = l.mixer, l.mixture
            f = {"kind": "dense", "ff": l.ffn_hidden_size} if l.ffn_hidden_size else None
            if x is not None:
                f = {"kind": "moe", "expert": {"ff": x.ff}, "router": {"experts": x.experts, "top": x.top}}
                if x.shared_ff:
                    f["shared"] = {"ff": x.shared_ff}
            out.append({"type": m.kind, "mlp": f,
                        "mixer": {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "scale": m.scale}})
        return {"architecture": self.architecture, "layers": out, "norm": {"eps": self.norm_eps}, "vocab": self.vocab_size,
                "width": self.hidden_size}

    def _count(self, active: bool) -> int:
        H, n = self.hidden_size, self.vocab_size * self.hidden_size + 2 * self.hidden_size
        for l in self.layers:
            m, x = l.mixer, l.mixture
            n += H * (m.heads * m.dim + m.kv_rank + m.heads + m.heads * m.vdim) + m.kv_rank * (1 + m.heads * (m.dim + m.vdim)) + 3 * H
            n += 2 * H * l.ffn_hidden_size + (3 * H if l.ffn_hidden_size else 0)
            if x is not None:
                n += 3 * H * (x.ff * (x.top if active else x.experts) + x.shared_ff) + x.experts * (H + 1) + 3 * H
        return n

    def num_params(self) -> int:
        return self._count(False)

    def active_params(self) -> int:
        """Parameters that take part in one token's pass."""
        return self._count(True)


@dataclass
class FigudraConfig:
    """Figudra: softmax attention of two kinds (capped scores and an output gate, no positions; or normed, rotated queries and keys in
    a window with kept first tokens and a sink) and gated linear attention in any order, with a dense (gelu) or grouped
    mixture-of-experts feed-forward beside the mixer under one norm, a normed embedding and a separate head.  A layer may use
    another layer's tensors.  ``from_dict`` reads the model folder's config.json; the rank of the decay projection is that of its
    tensor (``shapes``: tensor name -> shape).  ``max_seq_len`` as in ``LanedraConfig``."""
    vocab_size: int
    hidden_size: int
    layers: list
    norm_eps: float
    max_seq_len: int = 32768

    architecture = "Figudra"
    embedding_scale = 1.0
    tie_embeddings = False

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            m, x = l.mixer, l.mixture
            if m.kind == "head_attention":
                if m.heads % m.kv_heads:
                    raise ValueError(f"layer {i}: {m.heads} heads do not divide over {m.kv_heads} kv heads")
                if m.rot is not None and (m.rot.dims % 2 or not 0 < m.rot.dims <= m.dim):
                    raise ValueError(f"layer {i}: cannot rotate {m.rot.dims} of {m.dim} entries")
            elif not 1 <= m.dim <= 512 or not 1 <= m.rank <= 768:
                raise ValueError(f"layer {i}: key channels per head {m.dim} or rank {m.rank} are not in 1 .. 512, 1 .. 768")
            if x is not None:
                if x.experts % x.groups or not 1 <= x.keep <= x.groups or not 1 <= x.top <= x.experts // x.groups * x.keep:
                    raise ValueError(f"layer {i}: cannot choose {x.top} of {x.experts} experts in {x.keep} of {x.groups} groups")
                if x.groups > 1 and (x.groups > 32 or x.experts > 1024 or x.top > 32):
                    raise ValueError(f"layer {i}: grouped routing takes up to 32 groups, 1024 experts and 32 of them per token")
            if l.weights_of is not None:
                j = l.weights_of
                if not 0 <= j < len(self.layers) or j == i or self.layers[j].weights_of is not None:
                    raise ValueError(f"layer {i}: layer {j} has no tensors to share")
                if (self.layers[j].mixer, self.layers[j].ffn_hidden_size, self.layers[j].mixture) != (m, l.ffn_hidden_size, x):
                    raise ValueError(f"layer {i}: layer {j}'s tensors have other sizes or constants")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def _attention(self):
        return [l.mixer for l in self.layers if l.mixer.kind == "head_attention"]

    @property
    def window(self) -> int:
        """As ``LanedraConfig.window``, the kept first tokens aside."""
        w = [m.window for m in self._attention]
        return 0 if not w or 0 in w else max(w)

    @property
    def keep_first(self) -> int:
        return max((m.keep_first for m in self._attention), default=0)

    @classmethod
    def from_dict(cls, d: dict, shapes=None, **extra) -> "FigudraConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            m, f, src = e["mixer"], e.get("mlp"), e.get("weights_of")
            seen = set()
            while src is not None and 0 <= src < len(d["layers"]) and d["layers"][src].get("weights_of") is not None and src not in seen:
                seen.add(src)                  # the layer at the end of the chain has the tensors
                src = d["layers"][src]["weights_of"]
            if e["type"] == "attention":
                t = m["q_temp"]
                if t["every"] != int(t["every"]):
                    raise ValueError(f"layer {i}: q_temp.every has to be whole")
                mix = HeadAttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), gate=True, softcap=float(m["softcap"]),
                                        temp_coef=float(t["coef"]), temp_every=int(t["every"]))
            elif e["type"] == "attention_2":
                r, k = m["rot"], m["mask"]
                rot = RotarySpec(int(r["dims"]), float(r["base"]), linear=float((r.get("scaling") or {}).get("factor", 1.0)))
                mix = HeadAttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), rot, qk_norm=True, window=k["size"],
                                        keep_first=k.get("keep_first") or 0, sink=True)
            elif e["type"] == "gla":
                a1 = (shapes or {}).get(f"l{i if src is None else src}.mix.a1")
                mix = GatedLinearSpec(m["heads"], m["dim"], m["vdim"], float(m["tau"]), *(() if a1 is None else (a1[0],)))
            else:
                raise ValueError(f"layer {i}: unknown mixer '{e['type']}'")
            kind = f.get("kind", "dense") if f else None
            if kind == "dense":
                layers.append(StackLayer(mix, f["ff"], weights_of=src))
            elif kind == "moe":
                r, sh = f["router"], f.get("shared")
                g = r.get("groups") or {"count": 1, "keep": 1}
                layers.append(StackLayer(mix, 0, MixtureSpec(r["experts"], r["top"], f["expert"]["ff"], sh["ff"] if sh else 0, bool(sh), "sigmoid",
                                                             g["count"], g["keep"], float(r["scale"])), src))
            elif kind is None:
                layers.append(StackLayer(mix, weights_of=src))
            else:
                raise ValueError(f"layer {i}: unknown feed-forward '{kind}'")
        return cls(vocab_size=d["vocab"], hidden_size=d["width"], layers=layers, norm_eps=float(d["norm"]["eps"]), **extra)

    def to_dict(self) -> dict:
        """The config.json form."""
        out = []
        for l in self.layers:
            m, x = l.mixer, l.mixture
            a = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
            kind = m.kind
            if kind == "gla":
                a["tau"] = m.tau
            else:
                a.update(kv_heads=m.kv_heads, scale=m.scale)
                if m.rot is None:
                    kind = "attention"
                    a.update(softcap=m.softcap, q_temp={"coef": m.temp_coef, "every": m.temp_every})
                else:
                    kind = "attention_2"
                    a.update(mask={"size": m.window, "keep_first": m.keep_first},
                             rot={"dims": m.rot.dims, "base": m.rot.base, "scaling": {"factor": m.rot.linear}})
            f = {"kind": "dense", "ff": l.ffn_hidden_size} if l.ffn_hidden_size else None
            if x is not None:
                f = {"kind": "moe", "expert": {"ff": x.ff},
                     "router": {"experts": x.experts, "top": x.top, "scale": x.scale, "groups": {"count": x.groups, "keep": x.keep}}}
                if x.shared_ff:
                    f["shared"] = {"ff": x.shared_ff}
            e = {"type": kind, "mixer": a, "mlp": f}
            if l.weights_of is not None:
                e["weights_of"] = l.weights_of
            out.append(e)
        return {"architecture": self.architecture, "layers": out, "norm": {"eps": self.norm_eps}, "vocab": self.vocab_size, "width": self.hidden_size}

    def _count(self, active: bool) -> int:
        H, n = self.hidden_size, 2 * self.vocab_size * self.hidden_size + 2 * self.hidden_size
        for l in self.layers:
            m, x = l.mixer, l.mixture
            if l.weights_of is not None and not active:
                continue
            if m.kind == "gla":
                n += H * (m.heads * (2 * m.dim + 3 * m.vdim) + m.rank) + m.heads * m.dim * (m.rank + 1) + m.vdim
            else:
                n += H * (m.dim * (m.heads + m.kv_heads) + m.vdim * (m.kv_heads + m.heads * (2 if m.gate else 1))) + (2 * m.dim if m.qk_norm else 0)
            n += H + 3 * H * l.ffn_hidden_size
            if x is not None:
                n += 3 * H * (x.ff * (x.top if active else x.experts) + x.shared_ff) + H * (x.experts + int(x.shared_gate))
        return n

    def num_params(self) -> int:
        return self._count(False)

    def active_params(self) -> int:
        """Parameters that take part in one token's pass (those of a layer that is run twice count twice)."""
        return self._count(True)


@dataclass
class ToderaxConfig:
    """Toderax: HGRN2, or chunked softmax attention (no positions, normed queries and keys, learnt sinks and temperatures) and retention side
    by side, in any order, each with a mixture of clamped experts or none, norms in groups, and a residual of several hyper-connected
    streams; a scaled embedding and a separate head.  ``from_dict`` reads the model folder's config.json; ``max_seq_len`` as in
    ``LanedraConfig``."""
    vocab_size: int
    hidden_size: int
    layers: list
    norm_eps: float
    norm_groups: int = 1
    streams: int = 1
    embedding_scale: float = 1.0
    max_seq_len: int = 32768

    architecture = "Toderax"
    tie_embeddings = False

    def __post_init__(self):
        if self.norm_groups < 1 or self.hidden_size % self.norm_groups:
            raise ValueError(f"a width of {self.hidden_size} does not divide into {self.norm_groups} groups")
        if not 1 <= self.streams <= 16:
            raise ValueError(f"{self.streams} streams are not in 1 .. 16")
        for i, l in enumerate(self.layers):
            x = l.mixture
            for m in mixers_of(l.mixer):
                if m.kind == "head_attention":
                    if m.heads % m.kv_heads:
                        raise ValueError(f"layer {i}: {m.heads} heads do not divide over {m.kv_heads} kv heads")
                    if m.chunk < 1:
                        raise ValueError(f"layer {i}: a chunk of {m.chunk} positions")
                elif not 1 <= m.dim <= 512:
                    raise ValueError(f"layer {i}: key channels per head {m.dim} are not in 1 .. 512")
                if m.kind == "retention":
                    if len(m.decay) != m.heads:
                        raise ValueError(f"layer {i}: {len(m.decay)} decays for {m.heads} heads")
                    if m.rot.dims % 2 or not 0 <= m.rot.dims <= m.dim:
                        raise ValueError(f"layer {i}: cannot rotate {m.rot.dims} of {m.dim} entries")
            if x is not None and not 1 <= x.top <= x.experts:
                raise ValueError(f"layer {i}: cannot choose {x.top} of {x.experts} experts")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def window(self) -> int:
        """Positions that any attention layer may still look at, the current one included; 0: there is no such layer."""
        return max((m.chunk for l in self.layers for m in mixers_of(l.mixer) if m.kind == "head_attention"), default=0)

    @classmethod
    def from_dict(cls, d: dict, **extra) -> "ToderaxConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            m, f = e["mixer"], e.get("mlp")
            if e["type"] == "hgrn2":
                mix = ForgetLinearSpec(m["heads"], m["dim"], m["vdim"])
            elif e["type"] == "parallel":
                a, b = m["left"], m["right"]
                r = b["rot"]
                mix = PairSpec(HeadAttentionSpec(a["heads"], a["kv_heads"], a["dim"], a["vdim"], float(a["scale"]), qk_norm=True, chunk=a["mask"]["size"],
                                                 bias=True, qk_weight=False, head_temp=True, head_sink=True),
                               RetentionSpec(b["heads"], b["dim"], b["vdim"], tuple(float(x) for x in b["decay"]),
                                             RotarySpec(int(r["dims"]), float(r["base"]))))
            else:
                raise ValueError(f"layer {i}: unknown mixer '{e['type']}'")
            if f is not None and f.get("kind", "moe") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward '{f['kind']}'")
            mixture = None
            if f is not None:
                r, x, sh = f["router"], f["expert"], f.get("shared")
                mixture = MixtureSpec(r["experts"], r["top"], x["ff"], sh["ff"] if sh else 0, score="softmax_all", act="clamped", limit=float(x["limit"]),
                                      shared_limit=float(sh["limit"]) if sh else 0.0)
            layers.append(StackLayer(mix, 0, mixture))
        return cls(vocab_size=d["vocab"], hidden_size=d["width"], layers=layers, norm_eps=float(d["norm"]["eps"]), norm_groups=int(d["norm"].get("groups", 1)),
                   streams=int(d.get("streams", 1)), embedding_scale=float(d["embedding"]["scale"]), **extra)

    def to_dict(self) -> dict:
        """The config.json form."""
        out = []
        for l in self.layers:
            m, x, f = l.mixer, l.mixture, None
            if m.kind == "pair":
                a, b = m.left, m.right
                mix = {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale, "mask": {"size": a.chunk}},
                       "right": {"heads": b.heads, "dim": b.dim, "vdim": b.vdim, "decay": list(b.decay), "rot": {"dims": b.rot.dims, "base": b.rot.base}}}
            else:
                mix = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
            if x is not None:
                f = {"kind": "moe", "expert": {"ff": x.ff, "limit": x.limit}, "router": {"experts": x.experts, "top": x.top}}
                if x.shared_ff:
                    f["shared"] = {"ff": x.shared_ff, "limit": x.shared_limit}
            out.append({"type": "parallel" if m.kind == "pair" else m.kind, "mixer": mix, "mlp": f})
        return {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale}, "layers": out,
                "norm": {"eps": self.norm_eps, "groups": self.norm_groups}, "streams": self.streams, "vocab": self.vocab_size, "width": self.hidden_size}

    def _count(self, active: bool) -> int:
        H, s, n = self.hidden_size, self.streams, 2 * self.vocab_size * self.hidden_size + self.hidden_size
        for l in self.layers:
            x, around = l.mixture, H + 2 * s + s * s
            n += l.mixer.params(H) + around
            if x is not None:
                n += 3 * H * (x.ff * (x.top if active else x.experts) + x.shared_ff) + H * x.experts + around
        return n

    def num_params(self) -> int:
        return self._count(False)

    def active_params(self) -> int:
        """Parameters that take part in one token's pass."""
        return self._count(True)


# Named shapes used by the benchmarks and tests.
def preset(name: str) -> TransformerConfig:
    name = name.lower()
    if name in ("llama-50m", "cfg2"):
        return TransformerConfig(vocab_size=32000, hidden_size=512, num_layers=8, num_heads=8, ffn_hidden_size=1408,
                                 rope_theta=10000.0, max_seq_len=1024, activation="swiglu", tie_embeddings=True)
    if name in ("llama-3-8b", "cfg3"):
        return TransformerConfig(vocab_size=128256, hidden_size=4096, num_layers=32, num_heads=32, num_kv_heads=8,
                                 ffn_hidden_size=14336, rope_theta=500000.0, max_seq_len=4096, activation="swiglu")
    if name in ("mixtral-8x7b", "cfg4"):
        return MoEConfig(vocab_size=32000, hidden_size=4096, num_layers=32, num_heads=32, num_kv_heads=8,
                         ffn_hidden_size=14336, rope_theta=1000000.0, max_seq_len=4096, activation="swiglu",
                         num_experts=8, top_k=2, load_balance_weight=0.01, expert_fp8=True)
    if name in ("gpt2-small", "cfg1"):
        return TransformerConfig(vocab_size=50257, hidden_size=768, num_layers=12, num_heads=12, ffn_hidden_size=3072,
                                 max_seq_len=1024, activation="gelu", norm_type="layernorm", position_type="learned",
                                 attention_bias=True, tie_embeddings=True)
    if name in ("lanedra-1.5b", "lanedra-8b"):
        # layer sizes of the dense models they stand beside (dense-1.5b, llama-3-8b): the same width, feed-forward, key / value
        # bytes per token of an attention layer and query rows; half of the layers are the delta rule, and every second
        # attention layer looks at the keys of the one before it
        H, heads, kv, ff, n, V, win = (2048, 16, 4, 5632, 24, 32000, 2048) if name == "lanedra-1.5b" else (4096, 32, 8, 14336, 32, 128256, 4096)
        rot = RotarySpec(64, 500000.0, 4.0, 8192)
        layers = []
        for i in range(n):
            if i % 2 == 0:
                mix = GatedDeltaSpec(heads, heads, 128, 128, 4)
            else:
                mix = DiffAttentionSpec(heads, kv, 64, 128, 64 ** -0.5, 0.5, rot, win, i - 2 if i % 4 == 3 else None)
            layers.append(StackLayer(mix, ff))
        return LanedraConfig(V, H, layers, 1e-5, 1.0, max_seq_len=32768)
    if name in ("tekenex-7b", "tekenex-8x7b"):
        # beside mixture-7b and mixtral-8x7b: the same width, query rows and experts, of which one (two of mixture-7b's) is shared;
        # the first layer is dense
        H, heads, n, V, mix, ff = (2048, 16, 24, 32000, MixtureSpec(62, 6, 704, 1408), 8448) if name == "tekenex-7b" else \
            (4096, 32, 32, 32000, MixtureSpec(7, 1, 14336, 14336), 43008)
        att = LatentAttentionSpec(heads, 128, 128, 512, 128 ** -0.5)
        return TekenexConfig(V, H, [StackLayer(att, 0 if i else ff, mix if i else None) for i in range(n)], 1e-5)
    if name in ("figudra-7b", "figudra-8x7b"):
        # beside mixture-7b and mixtral-8x7b: the same width, query and key / value rows and feed-forward work per token (one shared
        # expert among it); one layer in three of each mixer, the first one's feed-forward dense
        H, heads, kv, n, V, win, mix, ff = (2048, 16, 4, 24, 32000, 1024, MixtureSpec(62, 6, 704, 1408, True, "sigmoid", 2, 1, 1.5), 5632) \
            if name == "figudra-7b" else (4096, 32, 8, 32, 32000, 4096, MixtureSpec(7, 1, 14336, 14336, True, "sigmoid"), 28672)
        mixers = (HeadAttentionSpec(heads, kv, 128, 128, 128 ** -0.5, gate=True, softcap=50.0, temp_coef=0.1, temp_every=8192),
                  HeadAttentionSpec(heads, kv, 128, 128, 128 ** -0.5, RotarySpec(64, 500000.0, linear=4.0), True, window=win, keep_first=16, sink=True),
                  GatedLinearSpec(heads, 128, 128, 16.0))
        return FigudraConfig(V, H, [StackLayer(mixers[i % 3], 0 if i else ff, mix if i else None) for i in range(n)], 1e-5)
    if name in ("toderax-7b", "toderax-8x7b"):
        # beside figudra-7b and figudra-8x7b: the same width, heads, feed-forward work per token and one shared expert; two layers in three
        # with attention and retention side by side (each with half of the heads), one with HGRN2; two streams
        H, heads, kv, n, V, experts = (2048, 16, 4, 24, 32000, (62, 6, 704, 1408)) if name == "toderax-7b" else (4096, 32, 8, 32, 32000, (7, 1, 14336, 14336))
        mix = MixtureSpec(*experts, score="softmax_all", act="clamped", limit=7.0, shared_limit=7.0)
        h = heads // 2
        pair = PairSpec(HeadAttentionSpec(h, kv // 2, 128, 128, 128 ** -0.5, qk_norm=True, chunk=8192, bias=True, qk_weight=False, head_temp=True, head_sink=True),
                        RetentionSpec(h, 128, 128, tuple(1 - 2.0 ** (-5 - 5.0 * i / h) for i in range(h)), RotarySpec(128, 10000.0)))
        mixers = (pair, pair, ForgetLinearSpec(heads, 128, 128))
        return ToderaxConfig(V, H, [StackLayer(mixers[i % 3], 0, mix) for i in range(n)], 1e-5, 4, 2)
    if name == "mixture-7b":
        return MoEConfig(vocab_size=32000, hidden_size=2048, num_layers=24, num_heads=16, num_kv_heads=4, ffn_hidden_size=704, rope_theta=500000.0,
                         max_seq_len=32768, activation="swiglu", num_experts=64, top_k=8)
    if name == "dense-1.5b":
        return TransformerConfig(vocab_size=32000, hidden_size=2048, num_layers=24, num_heads=16, num_kv_heads=4, ffn_hidden_size=5632,
                                 rope_theta=500000.0, max_seq_len=32768, activation="swiglu")
    if name == "tiny":
        return TransformerConfig(vocab_size=256, hidden_size=128, num_layers=2, num_heads=2, ffn_hidden_size=256,
                                 max_seq_len=128)
    raise KeyError(name)
