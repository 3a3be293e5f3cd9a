// Gated delta rule (linear attention with a per-head state matrix) for prompts and for decoding.
//
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q            per head, S is [D, V] in fp32
//
// Kernels:
//   delta_prep   one block per (strip of 16 tokens, head): causal convolution of q, k and v over time (per channel, with the last
//                inputs of the previous step as history), silu, unit length of q and k per head, the decay g and the step
//                size beta, and the dot products k_i.k_j, q_i.k_j of every four tokens.  Everything it hands on is fp32.
//   delta_coef   per head and four tokens: those dot products times the decays between the tokens.
//   delta_scan   prompts.  The columns of S are independent recurrences that share k and q, so a group of TPC threads owns CPT
//                columns (D / TPC entries of each, in registers as packed fp32 pairs) and walks over the tokens four at a
//                time.  With S the state before the four tokens and G_i, R_ij the products of the decays up to token i and
//                between tokens j and i,
//                    u_i = beta_i (v_i - G_i S^T k_i - sum_{j<i} R_ij (k_i.k_j) u_j)
//                    o_i = G_i S^T q_i + sum_{j<=i} R_ij (q_i.k_j) u_j
//                    S  <- G_4 S + sum_j R_4j k_j u_j^T
//                which is the recurrence itself with its four reductions over D made one: all eight products with S are taken
//                from the same old state, so four tokens have one shuffle reduction on their critical path.  k, q, v and the
//                coefficients of the next tokens travel to shared memory (bulk copies) while the current ones are used; the
//                state never leaves the registers between tokens, and the arithmetic is fp32 FMA throughout.
//   delta_step   one token per sequence: one block per (sequence, head) streams the state through registers once (read,
//                two products, rank-one update, write) and applies the gated norm of the head's output.
//
// Layouts of the prepared arrays (Sp: rows per sequence, S rounded up to 4, or 1 when decoding; Dp: D rounded up to the
// register tile, tails zero; Vp: V rounded up to 4): q, k [B, G, Sp, Dp], v [B, H, Sp, Vp], decay, beta [B, H, Sp],
// pair [B, G, Sp / 4, 16] (decoding: [B, G], k.q), coef [B, H, Sp / 4, 32].
#include "tfb_elem.cuh"
#include "tfb_host.h"

namespace tfb {
TFB_BOUNDS_DEFINE(delta_rule)

// ------------------------------------------------------------------------------------------------
// preparation
// ------------------------------------------------------------------------------------------------
struct DeltaPrepArgs {
  const void* proj;       // [B*S, ld]: q (G D) | k (G D) | v (H V) | gate (H V) | b (H) | a (H)
  long long ld;
  const void* conv_w;     // [2 G D + H V, taps]
  void* conv_state;       // [slots, taps - 1, 2 G D + H V] inputs of the last taps - 1 tokens
  const int* state_slots; // [B]; negative: no history is read or kept
  const void *A_log, *dt_bias;  // [H]
  const int* lens;        // [B] tokens of each sequence in this call (null: S)
  float *q, *k, *v, *decay, *beta, *pair;
  int S, Sp, G, H, D, Dp, V, Vp, taps, has_past, nslots;
};

constexpr int PREP_STRIP = 16;   // tokens per block: four groups of four, one per warp

// the convolution's activation may be bf16-accurate when its inputs are bf16; the fp32 form is exact
template <class T> __device__ __forceinline__ float conv_silu(float x) { return silu_exact(x); }
template <> __device__ __forceinline__ float conv_silu<__nv_bfloat16>(float x) { return __fdividef(x, 1.f + __expf(-x)); }

// One channel over the strip's tokens s0 .. s0 + n - 1: convolution, silu, emit(token in strip, value).  TAPS > 0: the window
// moves through registers; TAPS = 0: any number of taps, inputs re-read.
template <class T, int TAPS, class Emit>
__device__ __forceinline__ void conv_channel(const DeltaPrepArgs& p, const T* __restrict__ x0, T* hist, bool past, int C, int c, int s0, int n,
                                             Emit emit) {
  const T* cw = static_cast<const T*>(p.conv_w) + (long long)c * p.taps;
  const T* xc = x0 + (long long)s0 * p.ld + c;          // token s0, channel c
  auto before = [&](int j) -> float {    // the input j tokens before s0; before the call's first token: history
    if (s0 >= j) return to_f(xc[-(long long)j * p.ld]);
    return past ? to_f(hist[(long long)(p.taps - 1 + s0 - j) * C + c]) : 0.f;
  };
  const T newest = xc[0];
  if constexpr (TAPS > 0) {
    float w[TAPS], win[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = to_f(cw[j]);
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) win[j + 1] = before(TAPS - 1 - j);
    const T* xp = xc;
    for (int i0 = 0; i0 < n; i0 += 8) {
      T cur[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        cur[i] = i0 + i < n ? *xp : from_f<T>(0.f);
        xp += p.ld;
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) {
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) win[j] = win[j + 1];
        win[TAPS - 1] = to_f(cur[i]);
        float y = 0.f;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) y = fmaf(w[j], win[j], y);
        if (i0 + i < n) emit(i0 + i, conv_silu<T>(y));
      }
    }
  } else {
    for (int i = 0; i < n; ++i) {
      float y = 0.f;
      for (int j = 0; j < p.taps; ++j) {
        const int back = p.taps - 1 - j - i;          // tokens before s0; <= 0: in the strip
        y = fmaf(to_f(cw[j]), back > 0 ? before(back) : to_f(xc[-(long long)back * p.ld]), y);
      }
      emit(i, conv_silu<T>(y));
    }
  }
  if (p.S == 1 && hist) {                // decoding: this thread alone uses channel c, so the window moves in place
    const int m = p.taps - 1;
    for (int j = 0; j < m - 1; ++j) hist[(long long)j * C + c] = past ? hist[(long long)(j + 1) * C + c] : from_f<T>(0.f);
    hist[(long long)(m - 1) * C + c] = newest;
  }
}

// blockIdx.y < G: the q and k heads of group blockIdx.y; otherwise v and the gates of head blockIdx.y - G
template <class T, int TAPS>
__global__ void __launch_bounds__(128) delta_prep_kernel(const DeltaPrepArgs p) {
  tfb::pdl_sync();
  extern __shared__ float sqk[];         // [rows][2 Dp]; rows: the strip's, or 4 when decoding
  const int s0 = blockIdx.x * PREP_STRIP, b = blockIdx.z, tid = threadIdx.x, unit = blockIdx.y;
  const int len = p.lens ? p.lens[b] : p.S;
  const int len4 = p.Sp == 1 ? len : (len + 3) / 4 * 4;       // rows len .. len4 - 1 become tokens that change nothing
  if (s0 >= len4) return;
  const int n = max(0, min(PREP_STRIP, len - s0)), n4 = min(PREP_STRIP, len4 - s0);
  const T* x0 = static_cast<const T*>(p.proj) + (long long)b * p.S * p.ld;
  const int C = 2 * p.G * p.D + p.H * p.V;
  int slot = p.state_slots ? p.state_slots[b] : -1;
  TFB_BOUNDS(slot < p.nslots, 71, slot, p.nslots);
  if (slot >= p.nslots) slot = -1;
  T* hist = (slot >= 0 && p.taps > 1) ? static_cast<T*>(p.conv_state) + (long long)slot * (p.taps - 1) * C : nullptr;
  const bool past = hist && p.has_past;
  if (unit >= p.G) {
    const int h = unit - p.G;
    float* vo = p.v + (((long long)b * p.H + h) * p.Sp + s0) * p.Vp;
    for (int j = tid; j < p.V; j += 128)
      conv_channel<T, TAPS>(p, x0, hist, past, C, 2 * p.G * p.D + h * p.V + j, s0, n, [&](int i, float y) { vo[i * p.Vp + j] = y; });
    for (int i = tid; i < (n4 - n) * p.Vp; i += 128) vo[n * p.Vp + i] = 0.f;
    if (tid < n4) {
      const long long o = ((long long)b * p.H + h) * p.Sp + s0 + tid;
      if (tid < n) {
        const T* gb = x0 + (long long)(s0 + tid) * p.ld + C + p.H * p.V;
        const float z = to_f(gb[p.H + h]) + to_f(static_cast<const T*>(p.dt_bias)[h]);
        const float sp = z > 20.f ? z : log1pf(expf(z));
        p.beta[o] = 1.f / (1.f + expf(-to_f(gb[h])));
        p.decay[o] = expf(-expf(to_f(static_cast<const T*>(p.A_log)[h])) * sp);
      } else {
        p.beta[o] = 0.f;
        p.decay[o] = 1.f;
      }
    }
    return;
  }
  const int g = unit, Dp = p.Dp, W = 2 * Dp;
  const int rows = (n4 + 3) / 4 * 4;
  if (p.D < Dp || n < rows)              // the tails of the rows, and rows without a token
    for (int i = tid; i < rows * W; i += 128)
      if (i / W >= n || i % Dp >= p.D) sqk[i] = 0.f;
  for (int d = tid; d < p.D; d += 128) {
    conv_channel<T, TAPS>(p, x0, hist, past, C, g * p.D + d, s0, n, [&](int i, float y) { sqk[i * W + d] = y; });
    conv_channel<T, TAPS>(p, x0, hist, past, C, (p.G + g) * p.D + d, s0, n, [&](int i, float y) { sqk[i * W + Dp + d] = y; });
  }
  __syncthreads();
  // one warp per four tokens: the 24 products of their q and k vectors (as they are), reduced so that lane x holds product x;
  // the unit lengths come from the diagonal and scale the others
  const int blk = tid >> 5, lane = tid & 31;
  if (blk * 4 >= n4) return;
  const float* base = sqk + blk * 4 * W;
  float pr[32];
#pragma unroll
  for (int i = 0; i < 32; ++i) pr[i] = 0.f;
  for (int d = lane; d < Dp; d += 32) {
    float q[4], k[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      q[i] = base[i * W + d];
      k[i] = base[i * W + Dp + d];
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {        // order of the products: see coef; then the squares of k (16-19) and of q (20-23)
#pragma unroll
      for (int j = 0; j < i; ++j) pr[i * (i - 1) / 2 + j] = fmaf(k[i], k[j], pr[i * (i - 1) / 2 + j]);
#pragma unroll
      for (int j = 0; j <= i; ++j) pr[6 + i * (i + 1) / 2 + j] = fmaf(q[i], k[j], pr[6 + i * (i + 1) / 2 + j]);
      pr[16 + i] = fmaf(k[i], k[i], pr[16 + i]);
      pr[20 + i] = fmaf(q[i], q[i], pr[20 + i]);
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {     // o values stay with each half
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float send = up ? pr[i] : pr[i + o], keep = up ? pr[i + o] : pr[i];
      pr[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  const float mine = pr[0];
  // lanes 16-19: 1 / |k_i|, lanes 20-23: 1 / (|q_i| sqrt(D))
  float r = 1.f / sqrtf(mine + 1e-6f);
  if (lane >= 20) r = r / sqrtf(float(p.D));
  float rk[4], rq[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    rk[i] = __shfl_sync(0xffffffffu, r, 16 + i);
    rq[i] = __shfl_sync(0xffffffffu, r, 20 + i);
  }
  const long long row0 = ((long long)b * p.G + g) * p.Sp + s0 + blk * 4;
  const int nr = min(4, n4 - blk * 4);
  for (int d = lane; d < Dp; d += 32)
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (i < nr) {
        p.q[(row0 + i) * Dp + d] = base[i * W + d] * rq[i];
        p.k[(row0 + i) * Dp + d] = base[i * W + Dp + d] * rk[i];
      }
  if (p.Sp == 1) {
    if (lane == 6) p.pair[(long long)b * p.G + g] = mine * rq[0] * rk[0];
    return;
  }
  if (lane < 16) {
    const int y = lane < 6 ? lane : lane - 6;
    int i, j;
    if (lane < 6) { i = y < 1 ? 1 : y < 3 ? 2 : 3; j = y - (i * (i - 1)) / 2; }
    else { i = y < 1 ? 0 : y < 3 ? 1 : y < 6 ? 2 : 3; j = y - (i * (i + 1)) / 2; }
    float f = 0.f, e = 0.f;
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      if (x == i) f = lane < 6 ? rk[x] : rq[x];
      if (x == j) e = rk[x];
    }
    p.pair[(((long long)b * p.G + g) * (p.Sp / 4) + s0 / 4 + blk) * 16 + lane] = mine * f * e;
  }
}

// after a prompt portion: the inputs of its last taps - 1 tokens become the history (shorter portions keep part of the old one)
template <class T>
__global__ void __launch_bounds__(256) conv_history_kernel(const DeltaPrepArgs p) {
  tfb::pdl_sync();
  const int b = blockIdx.y, C = 2 * p.G * p.D + p.H * p.V, m = p.taps - 1;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  const int slot = p.state_slots[b];
  if (c >= C || slot < 0 || slot >= p.nslots) return;
  const int len = p.lens ? p.lens[b] : p.S;
  const T* x = static_cast<const T*>(p.proj) + (long long)b * p.S * p.ld;
  T* hist = static_cast<T*>(p.conv_state) + (long long)slot * m * C;
  for (int j = 0; j < m; ++j) {                       // reads run ahead of writes: entry j comes from entry j + len or from x
    const int t = len - m + j;
    T v = from_f<T>(0.f);
    if (t >= 0) v = x[(long long)t * p.ld + c];
    else if (p.has_past) v = hist[(long long)(m + t) * C + c];
    hist[(long long)j * C + c] = v;
  }
}

// ------------------------------------------------------------------------------------------------
// coefficients of four tokens of one head: [0,6) beta_i R_ij (k_i.k_j), [6,16) R_ij (q_i.k_j), [16,20) beta_i,
// [20,24) beta_i G_i, [24,28) G_i, [28,32) R_4j
// ------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(128) delta_coef_kernel(const float* __restrict__ pair, const float* __restrict__ decay,
                                                         const float* __restrict__ beta, float* __restrict__ coef, const int* __restrict__ lens,
                                                         int B, int S, int Sp, int G, int H) {
  tfb::pdl_sync();
  const int nb = Sp / 4;
  const long long id = blockIdx.x * 128ll + threadIdx.x;
  if (id >= (long long)B * H * nb) return;
  const int blk = int(id % nb), h = int(id / nb % H), b = int(id / nb / H), g = h / (H / G);
  if (blk * 4 >= (lens ? lens[b] : S)) return;
  const float4 d4 = *reinterpret_cast<const float4*>(decay + ((long long)b * H + h) * Sp + blk * 4);
  const float4 b4 = *reinterpret_cast<const float4*>(beta + ((long long)b * H + h) * Sp + blk * 4);
  const float* pr = pair + (((long long)b * G + g) * nb + blk) * 16;
  const float d[4] = {d4.x, d4.y, d4.z, d4.w}, be[4] = {b4.x, b4.y, b4.z, b4.w};
  float R[4][4], c[32];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    R[j][j] = 1.f;
#pragma unroll
    for (int i = j + 1; i < 4; ++i) R[i][j] = R[i - 1][j] * d[i];
  }
  float Gi = 1.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    Gi *= d[i];
#pragma unroll
    for (int j = 0; j < i; ++j) c[i * (i - 1) / 2 + j] = be[i] * R[i][j] * pr[i * (i - 1) / 2 + j];
#pragma unroll
    for (int j = 0; j <= i; ++j) c[6 + i * (i + 1) / 2 + j] = R[i][j] * pr[6 + i * (i + 1) / 2 + j];
    c[16 + i] = be[i];
    c[20 + i] = be[i] * Gi;
    c[24 + i] = Gi;
    c[28 + i] = R[3][i];
  }
  float4* out = reinterpret_cast<float4*>(coef + id * 32);
#pragma unroll
  for (int i = 0; i < 8; ++i) out[i] = make_float4(c[4 * i], c[4 * i + 1], c[4 * i + 2], c[4 * i + 3]);
}

// ------------------------------------------------------------------------------------------------
// scan over a prompt
// ------------------------------------------------------------------------------------------------
struct DeltaScanArgs {
  const float *q, *k, *v, *coef;
  float* o;               // [B*S, H, V]
  float* state;           // [slots, H, D, V]
  const int* state_slots; // [B]
  const int* lens;        // [B] or null
  int S, Sp, G, H, D, V, Vp, has_past, nslots;
  int* status;
};

constexpr int SCAN_CHUNK = 16;   // tokens per shared-memory stage

// EPT: entries of one column per thread (a multiple of 4); TPC: threads per column group; CPT: columns per group (a power of
// two, 2 CPT <= TPC); Dp = EPT TPC.  Of a group's 2 CPT sets of products (S^T k and S^T q of each column, four tokens each) a
// shuffle reduction leaves one set with each thread (or with each TPC / (2 CPT) threads): bits of the thread index, from the
// top: column, then k or q.
template <int EPT, int TPC, int CPT>
__global__ void __launch_bounds__(128) delta_scan_kernel(const DeltaScanArgs p) {
  tfb::pdl_sync();
  extern __shared__ __align__(128) float sm[];
  constexpr int Dp = EPT * TPC, CPW = 32 / TPC * CPT, SETS = 2 * CPT, W = TPC / SETS;
  static_assert(SETS <= TPC && EPT % 4 == 0, "tile shape");
  const int tid = threadIdx.x, lane = tid & 31, cols = (blockDim.x >> 5) * CPW;
  const int h = blockIdx.y, b = blockIdx.z, g = h / (p.H / p.G), col0 = blockIdx.x * cols;
  const int t = lane % TPC, cl = (tid >> 5) * CPW + lane / TPC * CPT;      // first column of the group, within the block
  const int set = t / W, my_col = col0 + cl + (set >> 1);                   // the products this thread ends up with
  const bool is_q = set & 1;
  const int len = p.lens ? p.lens[b] : p.S;
  const int stage_f = 2 * SCAN_CHUNK * Dp + SCAN_CHUNK * cols + SCAN_CHUNK * 8;
  const uint32_t bar = smem_u32(sm + 2 * stage_f);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(sm + 2 * stage_f + 4);
  if (tid == 0) {
    mbar_init(bar, 1);
    mbar_init(bar + 8, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  for (int i = tid; i < 2 * stage_f; i += blockDim.x) sm[i] = 0.f;        // columns past V stay zero
  fence_proxy_async_smem();
  __syncthreads();
  const float* kb = p.k + ((long long)b * p.G + g) * p.Sp * Dp;
  const float* qb = p.q + ((long long)b * p.G + g) * p.Sp * Dp;
  const float* vb = p.v + ((long long)b * p.H + h) * p.Sp * p.Vp + col0;
  const float* cb = p.coef + ((long long)b * p.H + h) * (p.Sp / 4) * 32;
  const int nrow = (len + 3) / 4 * 4, nc = min(cols, p.Vp - col0);
  auto issue = [&](int c) {              // warp 0: the rows of chunk c (whole groups of four)
    const int s0 = c * SCAN_CHUNK, n = min(SCAN_CHUNK, nrow - s0);
    if (n <= 0 || tid >= 32) return;
    float* base = sm + (c & 1) * stage_f;
    const uint32_t br = bar + (c & 1) * 8;
    if (lane == 0) mbar_expect_tx(br, uint32_t(n) * (2 * Dp + nc + 8) * 4);
    __syncwarp();
    if (lane == 0) bulk_load(smem_u32(base), kb + (long long)s0 * Dp, n * Dp * 4, br);
    if (lane == 1) bulk_load(smem_u32(base + SCAN_CHUNK * Dp), qb + (long long)s0 * Dp, n * Dp * 4, br);
    if (lane == 2) bulk_load(smem_u32(base + 2 * SCAN_CHUNK * Dp + SCAN_CHUNK * cols), cb + (long long)s0 * 8, n * 32, br);
    if (lane >= 16 && lane - 16 < n)
      bulk_load(smem_u32(base + 2 * SCAN_CHUNK * Dp + (lane - 16) * cols), vb + (long long)(s0 + lane - 16) * p.Vp, nc * 4, br);
  };
  issue(0);
  issue(1);

  int slot = p.state_slots ? p.state_slots[b] : -1;
  TFB_BOUNDS(slot < p.nslots, 72, slot, p.nslots);
  if (slot >= p.nslots) slot = -1;
  float* S0 = slot >= 0 ? p.state + ((long long)slot * p.H + h) * p.D * p.V : nullptr;
  // entry d of a column sits with thread (d / 4) % TPC, register (d / 4) / TPC * 4 + d % 4
  u64 st[CPT][EPT / 2];
#pragma unroll
  for (int x = 0; x < CPT; ++x)
#pragma unroll
    for (int i = 0; i < EPT / 4; ++i) {
      float f[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = (i * TPC + t) * 4 + e, col = col0 + cl + x;
        f[e] = (S0 && p.has_past && col < p.V && d < p.D) ? S0[(long long)d * p.V + col] : 0.f;
      }
      st[x][2 * i] = pack2(f[0], f[1]);
      st[x][2 * i + 1] = pack2(f[2], f[3]);
    }

  const int nchunk = (len + SCAN_CHUNK - 1) / SCAN_CHUNK;
  const long long ostep = (long long)p.H * p.V;
  float* orow = p.o + ((long long)b * p.S * p.H + h) * p.V + my_col;
  const bool writer = is_q && t % W == 0 && my_col < p.V;
  for (int c = 0; c < nchunk; ++c) {
    if (!mbar_wait_warp(bar + (c & 1) * 8, (c >> 1) & 1, abort_flag, p.status, ST_TIMEOUT_FULL)) break;
    const float* base = sm + (c & 1) * stage_f;
    const float* sv = base + 2 * SCAN_CHUNK * Dp;
    const float* sc = sv + SCAN_CHUNK * cols;
    const int n = min(SCAN_CHUNK, len - c * SCAN_CHUNK);
#pragma unroll 1
    for (int r = 0; r < n; r += 4) {
      u64 kk[4][EPT / 2];
      float val[SETS][4];                // [2 column + (k: 0, q: 1)][token]
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const ulonglong2* sk = reinterpret_cast<const ulonglong2*>(base + (r + i) * Dp) + t;
        const ulonglong2* sq = reinterpret_cast<const ulonglong2*>(base + (SCAN_CHUNK + r + i) * Dp) + t;
        u64 qq[EPT / 2];
#pragma unroll
        for (int e = 0; e < EPT / 4; ++e) {
          const ulonglong2 a = sk[e * TPC], q = sq[e * TPC];
          kk[i][2 * e] = a.x;
          kk[i][2 * e + 1] = a.y;
          qq[2 * e] = q.x;
          qq[2 * e + 1] = q.y;
        }
#pragma unroll
        for (int x = 0; x < CPT; ++x) {
          u64 dk = mul2(st[x][0], kk[i][0]), dq = mul2(st[x][0], qq[0]);     // 8 CPT independent chains over the four tokens
#pragma unroll
          for (int e = 1; e < EPT / 2; ++e) {
            dk = fma2(st[x][e], kk[i][e], dk);
            dq = fma2(st[x][e], qq[e], dq);
          }
          const float2 a = unpack2(dk), q = unpack2(dq);
          val[2 * x][i] = a.x + a.y;
          val[2 * x + 1][i] = q.x + q.y;
        }
      }
#pragma unroll
      for (int o = TPC >> 1, m = SETS; o > 0; o >>= 1) {
        if (m > 1) {                     // halve the sets: keep those of this thread's half, send the others
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
      const float4* cf = reinterpret_cast<const float4*>(sc + r * 8);
      const float4 c0 = cf[0], c1 = cf[1], c2 = cf[2], c3 = cf[3], be = cf[4], bg = cf[5], gi = cf[6], r4 = cf[7];
      float u[4];                        // right in the threads that hold a k set
      {
        const float* vr = sv + r * cols + cl + (set >> 1);
        u[0] = fmaf(be.x, vr[0], -bg.x * val[0][0]);
        u[1] = fmaf(-c0.x, u[0], fmaf(be.y, vr[cols], -bg.y * val[0][1]));
        u[2] = fmaf(-c0.z, u[1], fmaf(-c0.y, u[0], fmaf(be.z, vr[2 * cols], -bg.z * val[0][2])));
        u[3] = fmaf(-c1.y, u[2], fmaf(-c1.x, u[1], fmaf(-c0.w, u[0], fmaf(be.w, vr[3 * cols], -bg.w * val[0][3]))));
      }
      const u64 g4 = pack2(gi.w, gi.w);
      float mine[4] = {0.f, 0.f, 0.f, 0.f};      // u of this thread's column
#pragma unroll
      for (int x = 0; x < CPT; ++x) {
        float w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          w[i] = __shfl_sync(0xffffffffu, u[i], (lane & ~(TPC - 1)) + 2 * x * W);
          if (CPT == 1 || (set >> 1) == x) mine[i] = w[i];
        }
        const u64 w0 = pack2(w[0] * r4.x, w[0] * r4.x), w1 = pack2(w[1] * r4.y, w[1] * r4.y);
        const u64 w2 = pack2(w[2] * r4.z, w[2] * r4.z), w3 = pack2(w[3] * r4.w, w[3] * r4.w);
#pragma unroll
        for (int e = 0; e < EPT / 2; ++e)
          st[x][e] = fma2(kk[3][e], w3, fma2(kk[2][e], w2, fma2(kk[1][e], w1, fma2(kk[0][e], w0, mul2(st[x][e], g4)))));
      }
      if (writer) {
        float* op = orow + (long long)(c * SCAN_CHUNK + r) * ostep;
        op[0] = fmaf(c1.z, mine[0], gi.x * val[0][0]);
        if (r + 1 < n) op[ostep] = fmaf(c2.x, mine[1], fmaf(c1.w, mine[0], gi.y * val[0][1]));
        if (r + 2 < n) op[2 * ostep] = fmaf(c2.w, mine[2], fmaf(c2.z, mine[1], fmaf(c2.y, mine[0], gi.z * val[0][2])));
        if (r + 3 < n)
          op[3 * ostep] = fmaf(c3.w, mine[3], fmaf(c3.z, mine[2], fmaf(c3.y, mine[1], fmaf(c3.x, mine[0], gi.w * val[0][3]))));
      }
    }
    __syncthreads();
    issue(c + 2);
  }
  if (*abort_flag) {                     // a copy never landed: the status word says so, the state is left alone
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) {}      // bounded wait for copies already issued
    return;
  }
  if (writer)                            // padding: numbers, since a weight of zero does not silence what is not one
    for (int s = len; s < p.S; ++s) orow[s * ostep] = 0.f;
  if (S0) {
#pragma unroll
    for (int x = 0; x < CPT; ++x)
#pragma unroll
      for (int i = 0; i < EPT / 4; ++i) {
        const float2 a = unpack2(st[x][2 * i]), c = unpack2(st[x][2 * i + 1]);
        const float f[4] = {a.x, a.y, c.x, c.y};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = (i * TPC + t) * 4 + e, col = col0 + cl + x;
          if (d < p.D && col < p.V) S0[(long long)d * p.V + col] = f[e];
        }
      }
  }
}

template <int EPT, int TPC, int CPT>
static int launch_scan_tile(const DeltaScanArgs& p, int B, int nw, cudaStream_t st) {
  constexpr int CPW = 32 / TPC * CPT;
  auto bytes = [](int w) { return (2 * (2 * SCAN_CHUNK * EPT * TPC + SCAN_CHUNK * w * CPW + SCAN_CHUNK * 8) + 8) * int(sizeof(float)); };
  if (nw < 1 || nw > 4 || (nw * CPW) % 4) return TFB_ERR_ARG;      // rows of v are copied in 16-byte pieces
  static DeviceOnce once;
  auto kern = delta_scan_kernel<EPT, TPC, CPT>;
  if (int e = ensure_dyn_smem(once, kern, bytes(4))) return e;
  const int cols = nw * CPW;
  launch_k(kern, dim3((p.V + cols - 1) / cols, p.H, B), nw * 32, bytes(nw), st, p);
  return int(cudaGetLastError());
}

// warps per block for CPT columns per group of TPC threads: at least four columns, and blocks for most of the SMs
static int scan_warps(const DeltaScanArgs& p, int B, int tpc, int cpt) {
  const int cpw = 32 / tpc * cpt;
  const long long warps = (long long)((p.V + cpw - 1) / cpw) * p.H * B;
  int nw = 4;
  while (nw > 1 && nw / 2 * cpw >= 4 && (nw * cpw > (p.V + 3) / 4 * 4 || (warps + nw - 1) / nw < 4 * sm_count() / 5)) nw >>= 1;
  return nw;
}

template <int EPT, int TPC>
static int launch_scan(const DeltaScanArgs& p, int B, cudaStream_t st) {
  // Four columns per group read k and q from shared memory a quarter as often; for few sequences two columns per group of twice
  // as many threads give each scheduler something to do (measured at D = V = 128: 1.34 against 1.59 ms for one sequence of
  // 8192 tokens with 16 heads, 0.40 ms per 8192 tokens for many).
  constexpr int CPW = 32 / TPC * 4;
  if ((long long)((p.V + CPW - 1) / CPW) * p.H * B >= 3ll * sm_count())
    return launch_scan_tile<EPT, TPC, 4>(p, B, scan_warps(p, B, TPC, 4), st);
  if constexpr (EPT >= 8 && TPC <= 16) return launch_scan_tile<EPT / 2, TPC * 2, 2>(p, B, scan_warps(p, B, TPC * 2, 2), st);
  else return launch_scan_tile<EPT, TPC, 2>(p, B, scan_warps(p, B, TPC, 2), st);
}

// ------------------------------------------------------------------------------------------------
// one token per sequence
// ------------------------------------------------------------------------------------------------
struct DeltaStepArgs {
  const float *q, *k, *v, *kq, *decay, *beta;   // Sp = 1 layouts: [B, G, Dp], [B, G, Dp], [B, H, Vp], [B, G], [B, H], [B, H]
  float* state;
  const int* state_slots;
  int G, H, D, Dp, V, Vp, has_past, nslots;
};

// 256 threads = 8 warps; warp w holds rows w, w + 8, ... (NR of them) of the state, lane l the columns 4 l .. 4 l + 3 of
// each 128-column part.  D <= 8 NR, V <= 128 CV, V % 4 == 0.
template <class T, int NR, int CV>
__global__ void __launch_bounds__(256) delta_step_kernel(const DeltaStepArgs p, const T* __restrict__ gate, long long ldg,
                                                         const T* __restrict__ w, T* __restrict__ out, long long ldo, float eps) {
  tfb::pdl_sync();
  constexpr int VM = 128 * CV;
  __shared__ float sk[8 * NR], sq[8 * NR], su[VM], red_k[8][VM], red_q[8][VM], red[32];
  const int h = blockIdx.x, b = blockIdx.y, g = h / (p.H / p.G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int slot = p.state_slots[b];
  TFB_BOUNDS(slot < p.nslots, 73, slot, p.nslots);
  if (slot >= p.nslots) slot = -1;
  float* S0 = slot >= 0 ? p.state + ((long long)slot * p.H + h) * p.D * p.V : nullptr;
  float4 s[NR][CV];
#pragma unroll
  for (int i = 0; i < NR; ++i)
#pragma unroll
    for (int c = 0; c < CV; ++c) {
      const int d = warp + 8 * i, j = c * 128 + lane * 4;
      s[i][c] = (S0 && p.has_past && d < p.D && j < p.V) ? *reinterpret_cast<const float4*>(S0 + (long long)d * p.V + j) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  for (int d = tid; d < 8 * NR; d += 256) {
    sk[d] = d < p.D ? p.k[((long long)b * p.G + g) * p.Dp + d] : 0.f;
    sq[d] = d < p.D ? p.q[((long long)b * p.G + g) * p.Dp + d] : 0.f;
  }
  const float dec = p.decay[(long long)b * p.H + h], bet = p.beta[(long long)b * p.H + h], kq = p.kq[(long long)b * p.G + g];
  __syncthreads();
#pragma unroll
  for (int c = 0; c < CV; ++c) {
    float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const float kd = sk[warp + 8 * i], qd = sq[warp + 8 * i];
      const float4 v = s[i][c];
      ak.x = fmaf(v.x, kd, ak.x); ak.y = fmaf(v.y, kd, ak.y); ak.z = fmaf(v.z, kd, ak.z); ak.w = fmaf(v.w, kd, ak.w);
      aq.x = fmaf(v.x, qd, aq.x); aq.y = fmaf(v.y, qd, aq.y); aq.z = fmaf(v.z, qd, aq.z); aq.w = fmaf(v.w, qd, aq.w);
    }
    *reinterpret_cast<float4*>(&red_k[warp][c * 128 + lane * 4]) = ak;
    *reinterpret_cast<float4*>(&red_q[warp][c * 128 + lane * 4]) = aq;
  }
  __syncthreads();
  float ov = 0.f;                       // VM <= 256: at most one column per thread
  if (tid < VM && tid < p.V) {
    float dk = 0.f, dq = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      dk += red_k[i][tid];
      dq += red_q[i][tid];
    }
    const float u = bet * (p.v[((long long)b * p.H + h) * p.Vp + tid] - dec * dk);
    su[tid] = u;
    ov = fmaf(dec, dq, kq * u);
  } else if (tid < VM) {
    su[tid] = 0.f;
  }
  const float rs = 1.f / sqrtf(block_add(ov * ov, red) / p.V + eps);   // its barriers also publish su
  if (tid < p.V) {
    const float gt = to_f(gate[(long long)b * ldg + h * p.V + tid]);
    out[(long long)b * ldo + h * p.V + tid] = from_f<T>(ov * rs * to_f(w[tid]) * silu_exact(gt));
  }
  if (!S0) return;
#pragma unroll
  for (int i = 0; i < NR; ++i)
#pragma unroll
    for (int c = 0; c < CV; ++c) {
      const int d = warp + 8 * i, j = c * 128 + lane * 4;
      if (d < p.D && j < p.V) {
        const float kd = sk[d];
        float4 v = s[i][c];
        v.x = fmaf(kd, su[j], dec * v.x);
        v.y = fmaf(kd, su[j + 1], dec * v.y);
        v.z = fmaf(kd, su[j + 2], dec * v.z);
        v.w = fmaf(kd, su[j + 3], dec * v.w);
        *reinterpret_cast<float4*>(S0 + (long long)d * p.V + j) = v;
      }
    }
}

template <class T>
static int launch_step(const DeltaStepArgs& p, int B, const void* gate, long long ldg, const void* w, void* out, long long ldo, float eps,
                       cudaStream_t st) {
  const T* gt = static_cast<const T*>(gate);
  const T* wt = static_cast<const T*>(w);
  T* ot = static_cast<T*>(out);
  const dim3 grid(p.H, B);
#define TFB_STEP(NR, CV) launch_k(delta_step_kernel<T, NR, CV>, grid, 256, 0, st, p, gt, ldg, wt, ot, ldo, eps)
  if (p.V <= 128) {
    if (p.D <= 32) TFB_STEP(4, 1);
    else if (p.D <= 64) TFB_STEP(8, 1);
    else if (p.D <= 128) TFB_STEP(16, 1);
    else TFB_STEP(32, 1);
  } else {
    if (p.D <= 64) TFB_STEP(8, 2);
    else TFB_STEP(16, 2);
  }
#undef TFB_STEP
  return int(cudaGetLastError());
}

}  // namespace tfb

using bf16 = __nv_bfloat16;

// entries per key head in the prepared arrays (0: the head size is not supported)
TFB_API int tfb_delta_padded_dim(int D) {
  for (int d = 32; d <= 512; d *= 2)
    if (D <= d) return d;
  return 0;
}

// Convolution, activation, unit lengths, gates and (Sp > 1) the coefficients of B sequences with S rows each, lens[b] of them
// real.  has_past: the history in conv_state belongs to these sequences (otherwise they start here and see zeros).
TFB_API int tfb_delta_prep(const void* proj, long long ld, const void* conv_w, void* conv_state, const int* state_slots, int nslots,
                           const void* A_log, const void* dt_bias, const int* lens, float* q, float* k, float* v, float* decay, float* beta,
                           float* pair, float* coef, int B, int S, int Sp, int G, int H, int D, int V, int taps, int has_past, int f32,
                           void* stream) {
  using namespace tfb;
  const int Dp = tfb_delta_padded_dim(D);
  if (B <= 0 || B > 65535 || S <= 0 || G <= 0 || H % G || G + H > 65535 || D <= 0 || V <= 0 || taps < 1) return TFB_ERR_ARG;
  if (Sp != 1 && (Sp != (S + 3) / 4 * 4 || !coef)) return TFB_ERR_ARG;
  if (Sp == 1 && S != 1) return TFB_ERR_ARG;
  if (!Dp) return TFB_ERR_LIMIT;
  DeltaPrepArgs p{proj, ld, conv_w, conv_state, state_slots, A_log, dt_bias, lens, q, k, v, decay, beta, pair,
                  S, Sp, G, H, D, Dp, V, (V + 3) / 4 * 4, taps, has_past, nslots};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 grid((Sp + PREP_STRIP - 1) / PREP_STRIP, G + H, B);
  const int smem = (Sp == 1 ? 4 : PREP_STRIP) * 2 * Dp * int(sizeof(float));     // at most 64 KB
#define TFB_PREP1(T, TAPS)                                                                 \
  {                                                                                       \
    static DeviceOnce once;                                                               \
    if (int e = ensure_dyn_smem(once, delta_prep_kernel<T, TAPS>, 64 * 1024)) return e;   \
    launch_k(delta_prep_kernel<T, TAPS>, grid, 128, smem, st, p);                         \
  }
#define TFB_PREP(T)                                                                       \
  switch (taps) {                                                                         \
    case 2: TFB_PREP1(T, 2) break;                                                    \
    case 3: TFB_PREP1(T, 3) break;                                                    \
    case 4: TFB_PREP1(T, 4) break;                                                    \
    default: TFB_PREP1(T, 0) break;                                                   \
  }
  if (f32) { TFB_PREP(float) } else { TFB_PREP(bf16) }
#undef TFB_PREP
#undef TFB_PREP1
  if (S > 1 && taps > 1 && state_slots) {
    const dim3 hg((2 * G * D + H * V + 255) / 256, B);
    if (f32) launch_k(conv_history_kernel<float>, hg, 256, 0, st, p);
    else launch_k(conv_history_kernel<bf16>, hg, 256, 0, st, p);
  }
  if (Sp > 1)
    launch_k(delta_coef_kernel, int(((long long)B * H * (Sp / 4) + 127) / 128), 128, 0, st, pair, decay, beta, coef, lens, B, S, Sp, G, H);
  return int(cudaGetLastError());
}

// The recurrence over the prepared rows (Sp > 1); o [B*S, H, V] fp32.
TFB_API int tfb_delta_scan(const float* q, const float* k, const float* v, const float* coef, float* o, float* state, const int* state_slots,
                           int nslots, const int* lens, int B, int S, int G, int H, int D, int V, int has_past, int* status, void* stream) {
  using namespace tfb;
  if (B <= 0 || B > 65535 || S <= 0 || G <= 0 || H % G || H > 65535 || D <= 0 || V <= 0) return TFB_ERR_ARG;
  DeltaScanArgs p{q, k, v, coef, o, state, state_slots, lens, S, (S + 3) / 4 * 4, G, H, D, V, (V + 3) / 4 * 4, has_past, nslots, status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  switch (tfb_delta_padded_dim(D)) {
    case 32: return launch_scan<4, 8>(p, B, st);
    case 64: return launch_scan<8, 8>(p, B, st);
    case 128: return launch_scan<16, 8>(p, B, st);
    case 256: return launch_scan<16, 16>(p, B, st);
    case 512: return launch_scan<16, 32>(p, B, st);
    default: return TFB_ERR_LIMIT;
  }
}

// One token for each of B sequences (prepared with Sp = 1), gated norm included.  Returns TFB_ERR_LIMIT for head sizes it
// does not hold in registers (the caller then takes the scan and the norm kernel).
TFB_API int tfb_delta_step(const float* q, const float* k, const float* v, const float* kq, const float* decay, const float* beta, float* state,
                           const int* state_slots, int nslots, const void* gate, long long ldg, const void* w, void* out, long long ldo, int B,
                           int G, int H, int D, int V, int has_past, float eps, int f32, void* stream) {
  using namespace tfb;
  if (B <= 0 || B > 65535 || G <= 0 || H % G || D <= 0 || V <= 0 || !state_slots) return TFB_ERR_ARG;
  if ((V & 3) || V > 256 || D > 256 || (V > 128 && D > 128)) return TFB_ERR_LIMIT;
  DeltaStepArgs p{q, k, v, kq, decay, beta, state, state_slots, G, H, D, tfb_delta_padded_dim(D), V, V, has_past, nslots};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return f32 ? launch_step<float>(p, B, gate, ldg, w, out, ldo, eps, st) : launch_step<bf16>(p, B, gate, ldg, w, out, ldo, eps, st);
}
