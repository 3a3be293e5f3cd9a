// Linear attention with a matrix state per head whose rows decay, for prompts and for decoding.
//
//   S <- diag(a) S + k v^T;   o = S^T q            per head, S is [D, V] in fp32
//
// Three sources of q, k and the decays a (entries of the key channels):
//   GATED       a = sigmoid(z)^(1/tau), z out of a low-rank projection; q is scaled by D^(-1/2)
//   FORGET      a = l + (1 - l) sigmoid(f + b) with a lower bound l per channel, k = 1 - a, q through silu
//   RETENTION   a fixed number per head; q and k rotated by their position, k scaled by D^(-1/2)
//
// Kernels:
//   gla_prep    one warp per (four tokens, head): q, k and the decays, and what the scan needs of four tokens.  With G_i and R_ij the
//               products of the decays up to token i and between tokens j and i (per channel),
//                   q'_i = G_i q_i,   k'_j = R_3j k_j,   G_3,   P_ij = sum over the channels of q_i R_ij k_j   (j <= i)
//               Every factor is a product of decays, at most one: nothing is divided, and a channel that forgets at once is
//               no special case.
//   gla_scan    prompts:  o_i = S^T q'_i + sum_{j<=i} P_ij v_j,   S <- diag(G_3) S + sum_j k'_j v_j^T,   which is the recurrence itself over four
//               tokens.  The columns of S are independent, so a group of TPC threads owns CPT columns (D / TPC entries of each, in
//               registers as packed fp32 pairs).  The sums over D are needed for the output alone: no reduction is on the
//               path from one state to the next.  The rows of the next tokens travel to shared memory (bulk copies) while the
//               current ones are used; fp32 FMA throughout.  Few sequences leave most of the device idle, so theirs are cut into
//               segments: a first pass over all but the last computes what each adds to the state and the product of its decays, the
//               second, with the start of a segment put together from those before it, everything else.
//   gla_step    one token per sequence: one block per (sequence, head) computes q, k and the decays, streams the state through registers
//               once (read, updated, written back), and applies the norm (with weight and gate, where there are some) to the output.
#include "tfb_elem.cuh"
#include "tfb_host.h"

namespace tfb {
TFB_BOUNDS_DEFINE(gated_linear)

enum GlaKind { GATED = 0, FORGET = 1, RETENTION = 2 };

struct GlaProj {
  const void* proj;       // [B*S, ld]: q (H D) | k, or the logits f (H D) | v (H V) | gate (H V), where there is one | a1 (rank), GATED
  long long ld;
  int H, D, V, gated;
  const void* bias;       // [H D], GATED and FORGET
  const void* a2;         // GATED: [H D, ld2]
  long long ld2;
  int rank;
  float tau;
  const void* lower;      // FORGET: [H D]
  const float* decay;     // RETENTION: [H]
  const float *cos_t, *sin_t;   // [max_pos, dims / 2]
  const int* positions;   // [B*S]
  int max_pos, dims;      // the first `dims` entries of a head are rotated, entry i with entry i + dims / 2
};

// sigmoid(z)^(1 / tau) = exp((min(z, 0) - ln(1 + x)) / tau), x = exp(-|z|).  ln(1 + x) = 2 atanh(u) with u = x / (2 + x) <= 1 / 3, by the
// odd series up to u^13 (the next term is below 2^-25 of the sum); accurate relative to itself, so slow decays keep their digits.
__device__ __forceinline__ float channel_decay(float z, float inv_tau) {
  const float x = expf(-fabsf(z));
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(2.f + x));
  const float u = x * r, y = u * u;
  float p = 1.f / 13.f;
  p = fmaf(p, y, 1.f / 11.f);
  p = fmaf(p, y, 1.f / 9.f);
  p = fmaf(p, y, 1.f / 7.f);
  p = fmaf(p, y, 1.f / 5.f);
  p = fmaf(p, y, 1.f / 3.f);
  p = fmaf(p, y, 1.f);
  return expf((fminf(z, 0.f) - 2.f * u * p) * inv_tau);
}

// entry d of head h, in a row with position pos, that starts at x: rotated
template <class T>
__device__ __forceinline__ float rotated(const GlaProj& g, const T* x, int d, int pos) {
  const float u = to_f(x[d]);
  if (d >= g.dims) return u;
  const int half = g.dims >> 1, i = d < half ? d : d - half;
  const float c = g.cos_t[(long long)pos * half + i], s = g.sin_t[(long long)pos * half + i];
  return d < half ? u * c - to_f(x[d + half]) * s : u * c + to_f(x[d - half]) * s;
}

__device__ __forceinline__ int checked_position(const GlaProj& g, long long row) {
  if (g.dims == 0) return 0;
  int pos = g.positions[row];
  TFB_BOUNDS(pos >= 0 && pos < g.max_pos, 61, pos, g.max_pos);
  return pos < 0 ? 0 : (pos >= g.max_pos ? g.max_pos - 1 : pos);
}

// q, k and the decay of channel d < D of head h, for FORGET and RETENTION
template <class T, int KIND>
__device__ __forceinline__ void channel_of(const GlaProj& g, const T* row, int h, int d, int pos, float scale, float& q, float& k, float& a) {
  const long long c = (long long)h * g.D + d, n = (long long)g.H * g.D;
  if constexpr (KIND == FORGET) {
    const float z = to_f(row[n + c]) + to_f(static_cast<const T*>(g.bias)[c]), l = to_f(static_cast<const T*>(g.lower)[c]);
    const float e = expf(-fabsf(z)), big = 1.f / (1.f + e), small = e * big;      // sigmoid(|z|), sigmoid(-|z|)
    q = silu_exact(to_f(row[c]));
    k = (1.f - l) * (z < 0.f ? big : small);
    a = fmaf(1.f - l, z < 0.f ? small : big, l);
  } else {
    const T* x = row + (long long)h * g.D;
    q = rotated<T>(g, x, d, pos);
    k = rotated<T>(g, x + n, d, pos) * scale;
    a = g.decay[h];
  }
}

// ------------------------------------------------------------------------------------------------
// preparation
// ------------------------------------------------------------------------------------------------
struct GlaPrepArgs {
  GlaProj g;
  const int* lens;                  // [B] tokens of each sequence in this call (null: S)
  float *q, *k, *v, *decay, *pair;  // [B, H, Sp, Dp] twice, [B, H, Sp, Vp], [B, H, Sp / 4, Dp], [B, H, Sp / 4, 16]
  int S, Sp, Dp, Vp;
  int vec;                          // rows of a2 can be read eight entries at a time
};

constexpr int PREP_WARPS = 4;

template <class T, int KIND>
__global__ void __launch_bounds__(PREP_WARPS * 32) gla_prep_kernel(const GlaPrepArgs p) {
  tfb::pdl_sync();
  extern __shared__ __align__(16) float s_a1[];       // [warp][4][rank rounded up to 8] rows of a1, zeros past the rank
  const GlaProj& g = p.g;
  const int blk = blockIdx.x * PREP_WARPS + (threadIdx.x >> 5), h = blockIdx.y, b = blockIdx.z, lane = threadIdx.x & 31;
  const int len = p.lens ? p.lens[b] : p.S, s0 = blk * 4, n = min(4, len - s0), r8 = KIND == GATED ? (g.rank + 7) / 8 * 8 : 0;
  if (n <= 0) return;
  int pos[4];
  const T* row[4];
#pragma unroll
  for (int i = 0; i < 4; ++i)           // tokens past the end read the last one's rows and are made to change nothing
    row[i] = static_cast<const T*>(g.proj) + ((long long)b * p.S + s0 + min(i, n - 1)) * g.ld;
#pragma unroll
  for (int i = 0; i < 4; ++i) pos[i] = KIND == RETENTION ? checked_position(g, (long long)b * p.S + s0 + min(i, n - 1)) : 0;
  float* a1 = s_a1 + (threadIdx.x >> 5) * 4 * r8;
#pragma unroll
  for (int i = 0; i < 4; ++i)
    for (int r = lane; r < r8; r += 32) a1[i * r8 + r] = r < g.rank ? to_f(row[i][2 * g.H * (g.D + g.V) + r]) : 0.f;
  __syncwarp();
  const long long hb = (long long)b * g.H + h;
  float* qo = p.q + (hb * p.Sp + s0) * p.Dp;
  float* ko = p.k + (hb * p.Sp + s0) * p.Dp;
  const float scale = 1.f / sqrtf(float(g.D)), inv_tau = KIND == GATED ? 1.f / g.tau : 0.f;
  float pr[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) pr[i] = 0.f;
  // two channels at a time: d0 and d0 + 32, or, where all entries turn, a pair that turns together
  const bool turns = KIND == RETENTION && g.dims == g.D && p.Dp == g.D;
  const int apart = turns ? g.D / 2 : 32, d_end = turns ? g.D / 2 : p.Dp, d_step = turns ? 32 : 64;
  for (int d0 = lane; d0 < d_end; d0 += d_step) {
    float z[2][4];                                    // logits of the decays (GATED), or the decays
    float q[2][4], k[2][4];
    const T* w[2];
    if (turns) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const T* x = row[i] + (long long)h * g.D + d0;
        const long long at = (long long)pos[i] * apart + d0, kk = (long long)g.H * g.D;
        const float c = g.cos_t[at], s = g.sin_t[at], q0 = to_f(x[0]), q1 = to_f(x[apart]), k0 = to_f(x[kk]) * scale, k1 = to_f(x[kk + apart]) * scale;
        const float f = i < n ? 1.f : 0.f;
        q[0][i] = f * (q0 * c - q1 * s);
        q[1][i] = f * (q1 * c + q0 * s);
        k[0][i] = f * (k0 * c - k1 * s);
        k[1][i] = f * (k1 * c + k0 * s);
        z[0][i] = z[1][i] = g.decay[h];
      }
    } else if constexpr (KIND != GATED) {
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int d = d0 + 32 * x;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          channel_of<T, KIND>(g, row[i], h, d < g.D ? d : 0, pos[i], scale, q[x][i], k[x][i], z[x][i]);
          if (d >= g.D || i >= n) q[x][i] = k[x][i] = 0.f;
        }
      }
    } else {
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int d = d0 + 32 * x;
        const bool on = d < g.D;
        const long long c = (long long)h * g.D + (on ? d : 0);
        w[x] = static_cast<const T*>(g.a2) + c * g.ld2;
        const float bias = to_f(static_cast<const T*>(g.bias)[c]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          z[x][i] = bias;
          q[x][i] = on && i < n ? to_f(row[i][c]) * scale : 0.f;
          k[x][i] = on && i < n ? to_f(row[i][(long long)g.H * g.D + c]) : 0.f;
        }
      }
      for (int r = 0; r < r8; r += 8) {
        float f[2][8];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          if (p.vec) load_n<8>(w[x] + r, f[x]);
          else {
#pragma unroll
            for (int e = 0; e < 8; ++e) f[x][e] = r + e < g.rank ? to_f(w[x][r + e]) : 0.f;
          }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          float y[8];
          load_n<8>(a1 + i * r8 + r, y);
#pragma unroll
          for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int e = 0; e < 8; ++e) z[x][i] = fmaf(f[x][e], y[e], z[x][i]);
        }
      }
    }
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int d = d0 + apart * x;
      if (d >= p.Dp) break;
      float G = 1.f, t[4];              // t[j] = R_ij k_j for the current i
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float a = i < n && d < g.D ? (KIND == GATED ? channel_decay(z[x][i], inv_tau) : z[x][i]) : 1.f;
        G *= a;
#pragma unroll
        for (int j = 0; j < i; ++j) t[j] *= a;
        t[i] = k[x][i];
#pragma unroll
        for (int j = 0; j <= i; ++j) pr[i * (i + 1) / 2 + j] = fmaf(q[x][i], t[j], pr[i * (i + 1) / 2 + j]);
        qo[i * p.Dp + d] = G * q[x][i];
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) ko[j * p.Dp + d] = t[j];
      p.decay[(hb * (p.Sp / 4) + blk) * p.Dp + d] = G;
    }
  }
#pragma unroll
  for (int i = 0; i < 16; ++i) pr[i] += __shfl_xor_sync(0xffffffffu, pr[i], 16);
#pragma unroll
  for (int o = 8; o > 0; o >>= 1) {     // o values stay with each half: lane x ends up with product x
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float send = up ? pr[i] : pr[i + o], keep = up ? pr[i + o] : pr[i];
      pr[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  if (lane < 16) p.pair[(hb * (p.Sp / 4) + blk) * 16 + lane] = pr[0];
  float* vo = p.v + (hb * p.Sp + s0) * p.Vp;
  const long long v0 = 2ll * g.H * g.D + (long long)h * g.V;
#pragma unroll
  for (int i = 0; i < 4; ++i)
    for (int j = lane; j < p.Vp; j += 32) vo[i * p.Vp + j] = i < n && j < g.V ? to_f(row[i][v0 + j]) : 0.f;
}

// ------------------------------------------------------------------------------------------------
// scan over a prompt
// ------------------------------------------------------------------------------------------------
struct GlaScanArgs {
  const float *q, *k, *v, *decay, *pair;
  float* o;               // [B*S, H, V]
  float* state;           // [slots, H, D, V]
  const int* state_slots; // [B]
  const int* lens;        // [B] or null
  int S, Sp, H, D, V, Vp, has_past, nslots;
  int* status;
  int seg, nseg;          // tokens of a segment (a multiple of GS_CHUNK), segments of a sequence
  float* part;            // nseg > 1: [B, nseg, H, D, V]: the state behind segment i, of itself alone but for segment 0; last: the first state
  float* prod;            // nseg > 1: [B, nseg - 1, H, Dp]: products of the decays of segment i
};

constexpr int GS_CHUNK = 16;   // tokens per shared-memory stage

// EPT: entries of one column per thread (a multiple of 4); TPC: threads per column group; CPT: columns per group (powers of two, CPT <=
// TPC); Dp = EPT TPC.  A shuffle reduction of the CPT columns' four sums each leaves one column with each TPC / CPT threads.
enum { WHOLE = 0, SEG_FIRST = 1, SEG_SECOND = 2 };     // sequences in one piece; the first pass over segments (states and decays only); the second

// CPT neighbouring entries of a row, `n` of them in range (vec: a multiple of CPT, and aligned)
template <int CPT>
__device__ __forceinline__ void load_columns(const float* row, int n, bool vec, float (&f)[CPT]) {
  if constexpr (CPT == 4) {
    if (vec) {
      const float4 u = n > 0 ? *reinterpret_cast<const float4*>(row) : make_float4(0.f, 0.f, 0.f, 0.f);
      f[0] = u.x, f[1] = u.y, f[2] = u.z, f[3] = u.w;
      return;
    }
  } else if constexpr (CPT == 2) {
    if (vec) {
      const float2 u = n > 0 ? *reinterpret_cast<const float2*>(row) : make_float2(0.f, 0.f);
      f[0] = u.x, f[1] = u.y;
      return;
    }
  }
#pragma unroll
  for (int x = 0; x < CPT; ++x) f[x] = x < n ? row[x] : 0.f;
}

template <int EPT, int TPC, int CPT, int PASS>
__global__ void __launch_bounds__(128, 2) gla_scan_kernel(const GlaScanArgs p) {
  constexpr bool FIRST = PASS == SEG_FIRST;
  tfb::pdl_sync();
  extern __shared__ __align__(128) float sm[];
  constexpr int Dp = EPT * TPC, CPW = 32 / TPC * CPT, W = TPC / CPT;
  static_assert(CPT <= TPC && EPT % 4 == 0, "tile shape");
  const int tid = threadIdx.x, lane = tid & 31, cols = (blockDim.x >> 5) * CPW;
  const int nz = PASS == WHOLE ? 1 : FIRST ? p.nseg - 1 : p.nseg, si = PASS == WHOLE ? 0 : blockIdx.z % nz;
  const int h = blockIdx.y, b = PASS == WHOLE ? blockIdx.z : blockIdx.z / nz, col0 = blockIdx.x * cols;
  const int t = lane % TPC, cl = (tid >> 5) * CPW + lane / TPC * CPT;      // first column of the group, within the block
  const int my_cl = cl + t / W, my_col = col0 + my_cl;                      // the column this thread ends up with
  // this segment: rows first .. first + len - 1 of the sequence, and padding up to `end`
  const int total = p.lens ? p.lens[b] : p.S, first = si * p.seg, len = max(0, min(total - first, p.seg)), end = min(p.S, first + p.seg);
  if (FIRST && len < p.seg) return;      // nothing comes behind it
  constexpr int KQ = GS_CHUNK * Dp, DEC = GS_CHUNK / 4 * Dp, PR = GS_CHUNK * 4;
  const int stage_f = 2 * KQ + DEC + PR + GS_CHUNK * cols;
  const uint32_t bar = smem_u32(sm + 2 * stage_f);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(sm + 2 * stage_f + 4);
  if (tid == 0) {
    mbar_init(bar, 1);
    mbar_init(bar + 8, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  for (int s = 0; s < 2; ++s)                                              // columns of v past V stay zero
    for (int i = tid; i < GS_CHUNK * cols; i += blockDim.x) sm[s * stage_f + 2 * KQ + DEC + PR + i] = 0.f;
  fence_proxy_async_smem();
  __syncthreads();
  const long long hb = (long long)b * p.H + h;
  const float* qb = p.q + (hb * p.Sp + first) * Dp;
  const float* kb = p.k + (hb * p.Sp + first) * Dp;
  const float* db = p.decay + (hb * (p.Sp / 4) + first / 4) * Dp;
  const float* pb = p.pair + (hb * (p.Sp / 4) + first / 4) * 16;
  const float* vb = p.v + (hb * p.Sp + first) * p.Vp + col0;
  const int nrow = (len + 3) / 4 * 4, nc = min(cols, p.Vp - col0);
  auto issue = [&](int c) {              // warp 0: the rows of chunk c (whole groups of four)
    const int s0 = c * GS_CHUNK, n = min(GS_CHUNK, nrow - s0);
    if (n <= 0 || tid >= 32) return;
    float* base = sm + (c & 1) * stage_f;
    const uint32_t br = bar + (c & 1) * 8;
    if (lane == 0) mbar_expect_tx(br, uint32_t(n) * ((FIRST ? Dp : 2 * Dp + 4) + Dp / 4 + nc) * 4);
    __syncwarp();
    if (lane == 0 && !FIRST) bulk_load(smem_u32(base), qb + (long long)s0 * Dp, n * Dp * 4, br);
    if (lane == 1) bulk_load(smem_u32(base + KQ), kb + (long long)s0 * Dp, n * Dp * 4, br);
    if (lane == 2) bulk_load(smem_u32(base + 2 * KQ), db + (long long)(s0 / 4) * Dp, n * Dp, br);
    if (lane == 3 && !FIRST) bulk_load(smem_u32(base + 2 * KQ + DEC), pb + (long long)s0 * 4, n * 16, br);
    if (lane >= 16 && lane - 16 < n)
      bulk_load(smem_u32(base + 2 * KQ + DEC + PR + (lane - 16) * cols), vb + (long long)(s0 + lane - 16) * p.Vp, nc * 4, br);
  };
  issue(0);
  issue(1);

  int slot = p.state_slots ? p.state_slots[b] : -1;
  TFB_BOUNDS(slot < p.nslots, 72, slot, p.nslots);
  if (slot >= p.nslots) slot = -1;
  float* S0 = slot >= 0 ? p.state + ((long long)slot * p.H + h) * p.D * p.V : nullptr;
  const long long DV = (long long)p.D * p.V;
  auto part_of = [&](int i) { return p.part + (((long long)b * p.nseg + i) * p.H + h) * DV; };
  const float* start = nullptr;
  if (p.has_past && si == 0 && S0) start = PASS != SEG_SECOND || total < p.seg ? S0 : part_of(p.nseg - 1);
  const int nv = p.V - (col0 + cl);        // columns of this group that there are
  const bool vec = p.V % CPT == 0;
  // entry d of a column sits with thread (d / 4) % TPC, register (d / 4) / TPC * 4 + d % 4
  u64 st[CPT][EPT / 2];
  if constexpr (PASS == WHOLE) {
#pragma unroll
    for (int x = 0; x < CPT; ++x)
#pragma unroll
      for (int i = 0; i < EPT / 4; ++i) {
        float f[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = (i * TPC + t) * 4 + e, col = col0 + cl + x;
          f[e] = (start && col < p.V && d < p.D) ? start[(long long)d * p.V + col] : 0.f;
        }
        st[x][2 * i] = pack2(f[0], f[1]);
        st[x][2 * i + 1] = pack2(f[2], f[3]);
      }
  } else {
#pragma unroll
    for (int i = 0; i < EPT / 2; ++i) {
      float f[2][CPT];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = (i / 2 * TPC + t) * 4 + i % 2 * 2 + e, n = d < p.D ? nv : 0;
        const long long at = (long long)d * p.V + col0 + cl;
#pragma unroll
        for (int x = 0; x < CPT; ++x) f[e][x] = 0.f;
        if (start) load_columns<CPT>(start + at, n, vec, f[e]);
        if (FIRST && start) {                // the second pass may find it overwritten
#pragma unroll
          for (int x = 0; x < CPT; ++x)
            if (x < n) part_of(p.nseg - 1)[at + x] = f[e][x];
        }
        if (PASS == SEG_SECOND && len > 0 && n > 0) {
          for (int j = 0; j < si; ++j) {
            const float g = j ? p.prod[(((long long)b * (p.nseg - 1) + j) * p.H + h) * Dp + d] : 0.f;
            float u[CPT];
            load_columns<CPT>(part_of(j) + at, n, vec, u);
#pragma unroll
            for (int x = 0; x < CPT; ++x) f[e][x] = fmaf(g, f[e][x], u[x]);
          }
        }
      }
#pragma unroll
      for (int x = 0; x < CPT; ++x) st[x][i] = pack2(f[0][x], f[1][x]);
    }
  }
  u64 all[FIRST ? EPT / 2 : 1];          // products of the decays
#pragma unroll
  for (int i = 0; i < (FIRST ? EPT / 2 : 1); ++i) all[i] = pack2(1.f, 1.f);

  const int nchunk = (len + GS_CHUNK - 1) / GS_CHUNK;
  const long long ostep = (long long)p.H * p.V;
  float* orow = p.o + (((long long)b * p.S + first) * p.H + h) * p.V + my_col;
  const bool writer = t % W == 0 && my_col < p.V;
  for (int c = 0; c < nchunk; ++c) {
    if (!mbar_wait_warp(bar + (c & 1) * 8, (c >> 1) & 1, abort_flag, p.status, ST_TIMEOUT_FULL)) break;
    const float* base = sm + (c & 1) * stage_f;
    const float* sp = base + 2 * KQ + DEC;
    const float* sv = sp + PR;
    const int n = min(GS_CHUNK, len - c * GS_CHUNK);
#pragma unroll 1
    for (int r = 0; r < n; r += 4) {
      u64 acc[CPT][4], vv[CPT][4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int x = 0; x < CPT; ++x) {
          const float w = sv[(r + i) * cols + cl + x];
          vv[x][i] = pack2(w, w);
          acc[x][i] = pack2(0.f, 0.f);
        }
      const ulonglong2* sq = reinterpret_cast<const ulonglong2*>(base + r * Dp) + t;
      const ulonglong2* sk = reinterpret_cast<const ulonglong2*>(base + KQ + r * Dp) + t;
      const ulonglong2* sg = reinterpret_cast<const ulonglong2*>(base + 2 * KQ + r / 4 * Dp) + t;
#pragma unroll
      for (int e = 0; e < EPT / 4; ++e) {
        ulonglong2 q[4], k[4];
        const ulonglong2 g = sg[e * TPC];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if (!FIRST) q[i] = sq[i * (Dp / 4) + e * TPC];
          k[i] = sk[i * (Dp / 4) + e * TPC];
        }
        if constexpr (FIRST) {
          all[2 * e] = mul2(all[2 * e], g.x);
          all[2 * e + 1] = mul2(all[2 * e + 1], g.y);
        }
#pragma unroll
        for (int x = 0; x < CPT; ++x) {
          const u64 s0 = st[x][2 * e], s1 = st[x][2 * e + 1];
          if constexpr (!FIRST) {
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[x][i] = fma2(s1, q[i].y, fma2(s0, q[i].x, acc[x][i]));
          }
          u64 u0 = mul2(s0, g.x), u1 = mul2(s1, g.y);
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            u0 = fma2(k[i].x, vv[x][i], u0);
            u1 = fma2(k[i].y, vv[x][i], u1);
          }
          st[x][2 * e] = u0;
          st[x][2 * e + 1] = u1;
        }
      }
      if constexpr (!FIRST) {
        float val[CPT][4];
#pragma unroll
        for (int x = 0; x < CPT; ++x)
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float2 f = unpack2(acc[x][i]);
            val[x][i] = f.x + f.y;
          }
#pragma unroll
        for (int o = TPC >> 1, m = CPT; o > 0; o >>= 1) {
          if (m > 1) {                     // halve the columns: keep those of this thread's half, send the others
            const bool up = t & o;
#pragma unroll
            for (int y = 0; y < m / 2; ++y)
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                const float send = up ? val[y][i] : val[y + m / 2][i], keep = up ? val[y + m / 2][i] : val[y][i];
                val[y][i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
              }
            m >>= 1;
          } else {
#pragma unroll
            for (int i = 0; i < 4; ++i) val[0][i] += __shfl_xor_sync(0xffffffffu, val[0][i], o);
          }
        }
        if (writer) {
          const float4* pp = reinterpret_cast<const float4*>(sp + r * 4);
          const float4 p0 = pp[0], p1 = pp[1], p2 = pp[2];                   // (0,0) (1,0) (1,1) (2,0) | (2,1) (2,2) (3,0) (3,1) | (3,2) (3,3)
          const float* vr = sv + r * cols + my_cl;
          const float v0 = vr[0], v1 = vr[cols], v2 = vr[2 * cols], v3 = vr[3 * cols];
          float* op = orow + (long long)(c * GS_CHUNK + r) * ostep;
          op[0] = fmaf(p0.x, v0, val[0][0]);
          if (r + 1 < n) op[ostep] = fmaf(p0.z, v1, fmaf(p0.y, v0, val[0][1]));
          if (r + 2 < n) op[2 * ostep] = fmaf(p1.y, v2, fmaf(p1.x, v1, fmaf(p0.w, v0, val[0][2])));
          if (r + 3 < n) op[3 * ostep] = fmaf(p2.y, v3, fmaf(p2.x, v2, fmaf(p1.w, v1, fmaf(p1.z, v0, val[0][3]))));
        }
      }
    }
    __syncthreads();
    fence_proxy_async_smem();
    issue(c + 2);
  }
  if (*abort_flag) {                     // a copy never landed: the status word says so, the state is left alone
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) {}      // bounded wait for copies already issued
    return;
  }
  if (!FIRST && writer)                  // padding: numbers, since a weight of zero does not silence what is not one
    for (int s = len; s < end - first; ++s) orow[s * ostep] = 0.f;
  float* out = FIRST ? part_of(si) : (total > first || si == 0) && total <= first + p.seg ? S0 : nullptr;
  if (out) {
#pragma unroll
    for (int x = 0; x < CPT; ++x)
#pragma unroll
      for (int i = 0; i < EPT / 4; ++i) {
        const float2 a = unpack2(st[x][2 * i]), c = unpack2(st[x][2 * i + 1]);
        const float f[4] = {a.x, a.y, c.x, c.y};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = (i * TPC + t) * 4 + e, col = col0 + cl + x;
          if (d < p.D && col < p.V) out[(long long)d * p.V + col] = f[e];
        }
      }
  }
  if constexpr (FIRST) {
    if (blockIdx.x == 0 && tid < TPC) {
      float* g = p.prod + (((long long)b * (p.nseg - 1) + si) * p.H + h) * Dp;
#pragma unroll
      for (int i = 0; i < EPT / 4; ++i) {
        const float2 a = unpack2(all[2 * i]), c = unpack2(all[2 * i + 1]);
        *reinterpret_cast<float4*>(g + (i * TPC + t) * 4) = make_float4(a.x, a.y, c.x, c.y);
      }
    }
  }
}

template <int EPT, int TPC, int CPT>
static int launch_scan_tile(const GlaScanArgs& p, int B, cudaStream_t st) {
  constexpr int CPW = 32 / TPC * CPT;
  auto bytes = [](int w) { return (2 * (2 * GS_CHUNK * EPT * TPC + GS_CHUNK / 4 * EPT * TPC + GS_CHUNK * 4 + GS_CHUNK * w * CPW) + 8) * int(sizeof(float)); };
  // warps per block: rows of v are copied in 16-byte pieces, so at least four columns; blocks for most of the SMs
  const long long warps = (long long)((p.V + CPW - 1) / CPW) * p.H * B * p.nseg;
  int nw = 4;
  while (nw > 1 && nw / 2 * CPW >= 4 && (nw * CPW > p.Vp || (warps + nw - 1) / nw < 4 * sm_count() / 5)) nw >>= 1;
  if ((nw * CPW) % 4) return TFB_ERR_ARG;
  static DeviceOnce once, once_first, once_second;
  const int cols = nw * CPW;
  const unsigned gx = (p.V + cols - 1) / cols;
  if (p.nseg == 1) {
    auto kern = gla_scan_kernel<EPT, TPC, CPT, WHOLE>;
    if (int e = ensure_dyn_smem(once, kern, bytes(4))) return e;
    launch_k(kern, dim3(gx, p.H, B), nw * 32, bytes(nw), st, p);
    return int(cudaGetLastError());
  }
  auto first = gla_scan_kernel<EPT, TPC, CPT, SEG_FIRST>, second = gla_scan_kernel<EPT, TPC, CPT, SEG_SECOND>;
  if (int e = ensure_dyn_smem(once_first, first, bytes(4))) return e;
  if (int e = ensure_dyn_smem(once_second, second, bytes(4))) return e;
  launch_k(first, dim3(gx, p.H, B * (p.nseg - 1)), nw * 32, bytes(nw), st, p);
  launch_k(second, dim3(gx, p.H, B * p.nseg), nw * 32, bytes(nw), st, p);
  return int(cudaGetLastError());
}

// Warps of the form with four columns per group, the one that reads q' and k' from shared memory least often
static long long scan_warps(int B, int H, int Dp, int V) {
  const int TPC = Dp <= 128 ? 8 : Dp / 16, CPW = 32 / TPC * 4;
  return (long long)((V + CPW - 1) / CPW) * H * B;
}

template <int EPT, int TPC>
static int launch_scan(const GlaScanArgs& p, int B, cudaStream_t st) {
  // For few columns, two per group of twice as many threads give each scheduler something to do.
  if (scan_warps(B, p.H, EPT * TPC, p.V) * p.nseg >= 3ll * sm_count()) return launch_scan_tile<EPT, TPC, 4>(p, B, st);
  if constexpr (EPT >= 8 && TPC <= 16) return launch_scan_tile<EPT / 2, TPC * 2, 2>(p, B, st);
  else return launch_scan_tile<EPT, TPC, 2>(p, B, st);
}

// ------------------------------------------------------------------------------------------------
// one token per sequence
// ------------------------------------------------------------------------------------------------
struct GlaStepArgs {
  GlaProj g;
  float* state;
  const int* state_slots;
  int nslots, vec;
  const void* w;          // [V] weight of the norm, or null
  void* out;
  long long ldo;
  float eps;
};

// 256 threads = 8 warps; warp w holds rows w, w + 8, ... (NR of them) of the state, lane l the columns 4 l .. 4 l + 3 of each 128-column
// part.  D <= 8 NR, V <= 128 CV, V % 4 == 0.
template <class T, int KIND, int NR, int CV>
__global__ void __launch_bounds__(256, NR * CV <= 16 ? 2 : 1) gla_step_kernel(const GlaStepArgs p) {
  tfb::pdl_sync();
  constexpr int VM = 128 * CV;
  __shared__ float sk[8 * NR], sq[8 * NR], sa[8 * NR], sv[VM], so[8][VM], red[32];
  const GlaProj& g = p.g;
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, D = g.D, V = g.V;
  int slot = p.state_slots[b];
  TFB_BOUNDS(slot < p.nslots, 73, slot, p.nslots);
  if (slot >= p.nslots) slot = -1;
  float* S0 = slot >= 0 ? p.state + ((long long)slot * g.H + h) * D * V : nullptr;
  float4 s[NR][CV];
#pragma unroll
  for (int i = 0; i < NR; ++i)
#pragma unroll
    for (int c = 0; c < CV; ++c) {
      const int d = warp + 8 * i, j = c * 128 + lane * 4;
      s[i][c] = (S0 && d < D && j < V) ? *reinterpret_cast<const float4*>(S0 + (long long)d * V + j) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  const T* row = static_cast<const T*>(g.proj) + (long long)b * g.ld;
  const T* a1 = row + 2 * g.H * (D + V);
  const int pos = KIND == RETENTION ? checked_position(g, b) : 0;
  for (int d = tid; d < 8 * NR; d += 256) {
    float q = 0.f, k = 0.f, a = 1.f;
    if (KIND != GATED && d < D) channel_of<T, KIND>(g, row, h, d, pos, 1.f / sqrtf(float(D)), q, k, a);
    if (KIND == GATED && d < D) {
      const long long c = (long long)h * D + d;
      const T* w2 = static_cast<const T*>(g.a2) + c * g.ld2;
      float z = to_f(static_cast<const T*>(g.bias)[c]);
      if (p.vec) {
        for (int r = 0; r < g.rank; r += 8) {
          float x[8], y[8];
          load_n<8>(w2 + r, x);
          load_n<8>(a1 + r, y);
#pragma unroll
          for (int e = 0; e < 8; ++e) z = fmaf(x[e], y[e], z);
        }
      } else {
        for (int r = 0; r < g.rank; ++r) z = fmaf(to_f(w2[r]), to_f(a1[r]), z);
      }
      a = channel_decay(z, 1.f / g.tau);
      q = to_f(row[c]) / sqrtf(float(D));
      k = to_f(row[(long long)g.H * D + c]);
    }
    sq[d] = q;
    sk[d] = k;
    sa[d] = a;
  }
  const T* vrow = row + 2ll * g.H * D + (long long)h * V;
  for (int j = tid; j < VM; j += 256) sv[j] = j < V ? to_f(vrow[j]) : 0.f;
  __syncthreads();
#pragma unroll
  for (int c = 0; c < CV; ++c) {
    const float4 v = *reinterpret_cast<const float4*>(&sv[c * 128 + lane * 4]);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = warp + 8 * i, j = c * 128 + lane * 4;
      const float a = sa[d], k = sk[d], q = sq[d];
      float4 x = s[i][c];
      x.x = fmaf(a, x.x, k * v.x);
      x.y = fmaf(a, x.y, k * v.y);
      x.z = fmaf(a, x.z, k * v.z);
      x.w = fmaf(a, x.w, k * v.w);
      if (S0 && d < D && j < V) *reinterpret_cast<float4*>(S0 + (long long)d * V + j) = x;
      o.x = fmaf(x.x, q, o.x);
      o.y = fmaf(x.y, q, o.y);
      o.z = fmaf(x.z, q, o.z);
      o.w = fmaf(x.w, q, o.w);
    }
    *reinterpret_cast<float4*>(&so[warp][c * 128 + lane * 4]) = o;
  }
  __syncthreads();
  float ov = 0.f;                       // VM <= 256: at most one column per thread
  if (tid < V) {
#pragma unroll
    for (int i = 0; i < 8; ++i) ov += so[i][tid];
  }
  const float rs = 1.f / sqrtf(block_add(ov * ov, red) / V + p.eps);
  if (tid < V) {
    float y = ov * rs;
    if (p.w) y *= to_f(static_cast<const T*>(p.w)[tid]);
    if (g.gated) y *= silu_exact(to_f(vrow[(long long)g.H * V + tid]));
    static_cast<T*>(p.out)[(long long)b * p.ldo + h * V + tid] = from_f<T>(y);
  }
}

template <class T, int KIND>
static int launch_step(const GlaStepArgs& p, int B, cudaStream_t st) {
  const dim3 grid(p.g.H, B);
#define TFB_STEP(NR, CV) launch_k(gla_step_kernel<T, KIND, NR, CV>, grid, 256, 0, st, p)
  if (p.g.V <= 128) {
    if (p.g.D <= 32) TFB_STEP(4, 1);
    else if (p.g.D <= 64) TFB_STEP(8, 1);
    else if (p.g.D <= 128) TFB_STEP(16, 1);
    else TFB_STEP(32, 1);
  } else {
    if (p.g.D <= 64) TFB_STEP(8, 2);
    else TFB_STEP(16, 2);
  }
#undef TFB_STEP
  return int(cudaGetLastError());
}

static int padded_dim(int D) {
  for (int d = 32; d <= 512; d *= 2)
    if (D <= d) return d;
  return 0;
}

static int vector_rows(const GlaProj& g, int f32) {
  const int es = f32 ? 4 : 2, m = f32 ? 4 : 8;
  auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  const char* a1 = static_cast<const char*>(g.proj) + 2ll * g.H * (g.D + g.V) * es;
  return g.rank % 8 == 0 && g.ld % m == 0 && g.ld2 % m == 0 && al(a1) && al(g.a2);
}

// Launches of a source of q, k and decays (g, kind) with elements fp32 or bf16
static int run_prep(const GlaProj& g, int kind, const int* lens, float* q, float* k, float* v, float* decay, float* pair, int B, int S, int Dp, int f32,
                    void* stream) {
  if (B <= 0 || B > 65535 || S <= 0 || g.H <= 0 || g.H > 65535 || g.D <= 0 || g.V <= 0 || Dp != padded_dim(g.D)) return TFB_ERR_ARG;
  if (!Dp) return TFB_ERR_LIMIT;
  const GlaPrepArgs p{g, lens, q, k, v, decay, pair, S, (S + 3) / 4 * 4, Dp, (g.V + 3) / 4 * 4, kind == GATED && vector_rows(g, f32)};
  const dim3 grid((p.Sp / 4 + PREP_WARPS - 1) / PREP_WARPS, g.H, B);
  const int smem = kind == GATED ? PREP_WARPS * 4 * ((g.rank + 7) / 8 * 8) * 4 : 0;
  if (smem > 48 * 1024) return TFB_ERR_LIMIT;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define TFB_PREP(KIND)                                                                             \
  if (f32) launch_k(gla_prep_kernel<float, KIND>, grid, PREP_WARPS * 32, smem, st, p);             \
  else launch_k(gla_prep_kernel<__nv_bfloat16, KIND>, grid, PREP_WARPS * 32, smem, st, p);         \
  break
  switch (kind) {
    case GATED: TFB_PREP(GATED);
    case FORGET: TFB_PREP(FORGET);
    default: TFB_PREP(RETENTION);
  }
#undef TFB_PREP
  return int(cudaGetLastError());
}

// TFB_ERR_LIMIT for head sizes that the kernel does not hold in registers (the caller then takes the preparation, the scan and the norm)
static int run_step(const GlaProj& g, int kind, float* state, const int* state_slots, int nslots, const void* w, void* out, long long ldo, int B, float eps,
                    int f32, void* stream) {
  if (B <= 0 || B > 65535 || g.H <= 0 || g.D <= 0 || g.V <= 0 || !state_slots) return TFB_ERR_ARG;
  if ((g.V & 3) || g.V > 256 || g.D > 256 || (g.V > 128 && g.D > 128)) return TFB_ERR_LIMIT;
  const GlaStepArgs p{g, state, state_slots, nslots, kind == GATED && vector_rows(g, f32), w, out, ldo, eps};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  switch (kind) {
    case GATED: return f32 ? launch_step<float, GATED>(p, B, st) : launch_step<__nv_bfloat16, GATED>(p, B, st);
    case FORGET: return f32 ? launch_step<float, FORGET>(p, B, st) : launch_step<__nv_bfloat16, FORGET>(p, B, st);
    default: return f32 ? launch_step<float, RETENTION>(p, B, st) : launch_step<__nv_bfloat16, RETENTION>(p, B, st);
  }
}

static GlaProj gated_source(const void* proj, long long ld, const void* a2, long long ld2, const void* bias, int rank, float tau, int H, int D, int V) {
  GlaProj g{proj, ld, H, D, V, 1};
  g.bias = bias, g.a2 = a2, g.ld2 = ld2, g.rank = rank, g.tau = tau;
  return g;
}
static GlaProj forget_source(const void* proj, long long ld, const void* bias, const void* lower, int gated, int H, int D, int V) {
  GlaProj g{proj, ld, H, D, V, gated};
  g.bias = bias, g.lower = lower;
  return g;
}
static GlaProj retention_source(const void* proj, long long ld, const float* decay, const float* cos_t, const float* sin_t, int max_pos, int dims,
                                const int* positions, int gated, int H, int D, int V) {
  GlaProj g{proj, ld, H, D, V, gated};
  g.decay = decay, g.cos_t = cos_t, g.sin_t = sin_t, g.max_pos = max_pos, g.dims = dims, g.positions = positions;
  return g;
}
static bool bad_retention(const GlaProj& g) {
  return !g.decay || g.dims < 0 || (g.dims & 1) || g.dims > g.D || (g.dims && (!g.cos_t || !g.sin_t || !g.positions || g.max_pos <= 0));
}

}  // namespace tfb

// Preparation of the rows of B sequences for tfb_gla_scan; sources: see GlaProj; outputs: see GlaPrepArgs (Sp = S rounded up to 4, Dp: D
// rounded up to a power of two from 32 to 512).
TFB_API int tfb_gla_prep(const void* proj, long long ld, const void* a2, long long ld2, const void* bias, int rank, float tau, const int* lens,
                         float* q, float* k, float* v, float* decay, float* pair, int B, int S, int H, int D, int Dp, int V, int f32,
                         void* stream) {
  using namespace tfb;
  if (rank <= 0 || !(tau > 0.f)) return TFB_ERR_ARG;
  return run_prep(gated_source(proj, ld, a2, ld2, bias, rank, tau, H, D, V), GATED, lens, q, k, v, decay, pair, B, S, Dp, f32, stream);
}

TFB_API int tfb_forget_prep(const void* proj, long long ld, const void* bias, const void* lower, const int* lens, float* q, float* k, float* v,
                            float* decay, float* pair, int B, int S, int H, int D, int Dp, int V, int f32, void* stream) {
  using namespace tfb;
  if (!bias || !lower) return TFB_ERR_ARG;
  return run_prep(forget_source(proj, ld, bias, lower, 0, H, D, V), FORGET, lens, q, k, v, decay, pair, B, S, Dp, f32, stream);
}

TFB_API int tfb_retention_prep(const void* proj, long long ld, const float* head_decay, const float* cos_t, const float* sin_t, int max_pos, int dims,
                               const int* positions, const int* lens, float* q, float* k, float* v, float* decay, float* pair, int B, int S, int H, int D,
                               int Dp, int V, int f32, void* stream) {
  using namespace tfb;
  const GlaProj g = retention_source(proj, ld, head_decay, cos_t, sin_t, max_pos, dims, positions, 0, H, D, V);
  if (bad_retention(g)) return TFB_ERR_ARG;
  return run_prep(g, RETENTION, lens, q, k, v, decay, pair, B, S, Dp, f32, stream);
}

// Segments into which tfb_gla_scan cuts sequences of S tokens: as many as give the device enough warps, if the sequences alone give it less
// than half of them (the first pass costs about half of the second), of at least 256 tokens.
TFB_API int tfb_gla_scan_segments(int B, int S, int H, int D, int V) {
  using namespace tfb;
  if (B <= 0 || S <= 0 || H <= 0 || D <= 0 || V <= 0 || !padded_dim(D)) return 1;
  const long long warps = scan_warps(B, H, padded_dim(D), V), want = 6ll * sm_count();
  int n = 1;
  if (warps * 5 <= want * 2)
    while (n < 32 && warps * n < want && S / (2 * n) >= 256) n *= 2;
  return n;
}

// The recurrence over prepared rows; o [B*S, H, V] fp32.  segments > 1: every sequence is cut into (at most) so many, with work (fp32) of
// B segments H (D V + Dp) entries.
TFB_API int tfb_gla_scan(const float* q, const float* k, const float* v, const float* decay, const float* pair, float* o, float* state, int nslots,
                         const int* state_slots, int B, int S, int H, int D, int V, int has_past, const int* lens, int segments, float* work, int* status,
                         void* stream) {
  using namespace tfb;
  if (B <= 0 || B > 65535 || S <= 0 || H <= 0 || H > 65535 || D <= 0 || V <= 0 || segments < 1 || (segments > 1 && !work)) return TFB_ERR_ARG;
  const int seg = ((S + segments - 1) / segments + GS_CHUNK - 1) / GS_CHUNK * GS_CHUNK, nseg = (S + seg - 1) / seg;
  if ((long long)B * nseg > 65535) return TFB_ERR_LIMIT;
  const GlaScanArgs p{q, k, v, decay, pair, o, state, state_slots, lens, S, (S + 3) / 4 * 4, H, D, V, (V + 3) / 4 * 4, has_past, nslots, status, seg, nseg,
                      work ? work + (long long)B * (nseg - 1) * H * padded_dim(D) : nullptr, work};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  switch (padded_dim(D)) {
    case 32: return launch_scan<4, 8>(p, B, st);
    case 64: return launch_scan<8, 8>(p, B, st);
    case 128: return launch_scan<16, 8>(p, B, st);
    case 256: return launch_scan<16, 16>(p, B, st);
    case 512: return launch_scan<16, 32>(p, B, st);
    default: return TFB_ERR_LIMIT;
  }
}

// One token for each of B sequences that go on, with the norm of the heads' outputs: o / rms(o) [* w] [* silu(gate)].  TFB_ERR_LIMIT: see run_step.
TFB_API int tfb_gla_step(const void* proj, long long ld, const void* a2, long long ld2, const void* bias, int rank, float tau, float* state,
                         const int* state_slots, int nslots, const void* w, void* out, long long ldo, int B, int H, int D, int V, float eps, int f32,
                         void* stream) {
  using namespace tfb;
  if (rank <= 0 || !(tau > 0.f)) return TFB_ERR_ARG;
  return run_step(gated_source(proj, ld, a2, ld2, bias, rank, tau, H, D, V), GATED, state, state_slots, nslots, w, out, ldo, B, eps, f32, stream);
}

TFB_API int tfb_forget_step(const void* proj, long long ld, const void* bias, const void* lower, int gated, float* state, const int* state_slots, int nslots,
                            const void* w, void* out, long long ldo, int B, int H, int D, int V, float eps, int f32, void* stream) {
  using namespace tfb;
  if (!bias || !lower) return TFB_ERR_ARG;
  return run_step(forget_source(proj, ld, bias, lower, gated, H, D, V), FORGET, state, state_slots, nslots, w, out, ldo, B, eps, f32, stream);
}

TFB_API int tfb_retention_step(const void* proj, long long ld, const float* head_decay, const float* cos_t, const float* sin_t, int max_pos, int dims,
                               const int* positions, int gated, float* state, const int* state_slots, int nslots, const void* w, void* out,
                               long long ldo, int B, int H, int D, int V, float eps, int f32, void* stream) {
  using namespace tfb;
  const GlaProj g = retention_source(proj, ld, head_decay, cos_t, sin_t, max_pos, dims, positions, gated, H, D, V);
  if (bad_retention(g)) return TFB_ERR_ARG;
  return run_step(g, RETENTION, state, state_slots, nslots, w, out, ldo, B, eps, f32, stream);
}
