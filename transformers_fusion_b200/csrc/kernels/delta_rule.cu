// Gated delta rule (linear attention with a per-head state matrix) for prompts and for decoding.
//
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q            per head, S is [D, V] in fp32
//
// Kernels:
//   delta_prep   one block per (16 tokens, head): causal convolution of q, k and v over time (per channel, with the last inputs
//                of the previous step as history), silu, unit length of q and k per head, the decay g and the step size beta.
//                Everything it hands on is fp32.
//   delta_wy     prompts: one block per (16 tokens, head).  With S the state before the 16 tokens, G_i and R_ij the products of
//                the decays up to token i and between tokens j and i, the recurrence reads
//                    u_i = beta_i (v_i - G_i S^T k_i - sum_{j<i} R_ij (k_i.k_j) u_j)
//                    o_i = G_i S^T q_i + sum_{j<=i} R_ij (q_i.k_j) u_j
//                    S  <- G_last S + sum_j R_last,j k_j u_j^T
//                The triangular system for u does not need S: forward substitution turns beta v and beta G k into rows y and w
//                with u_i = y_i - S^T w_i.
//   delta_scan   prompts: what is left of the recurrence, 16 tokens at a time.  The columns of S are independent, so a group
//                of TPC threads owns CPT columns (D / TPC entries of each, in registers as packed fp32 pairs): 32 products with
//                the old state, one shuffle reduction, u, o, and the update.  The rows of the next 16 tokens travel to shared
//                memory (bulk copies) meanwhile; the state never leaves the registers between tokens.
//   delta_step   decoding: one block per (sequence, head) streams the state through registers once (read, two products,
//                rank-one update, write) and applies the gated norm of the head's output.
// All of it is fp32 FMA arithmetic.
//
// Layouts of the prepared arrays (Sp: rows per sequence, S rounded up to 16, or 1 when decoding; Dp: D rounded up to the
// register tile, tails zero; Vp: V rounded up to 4): q, k [B, G, Sp, Dp], v (later y) [B, H, Sp, Vp], w [B, H, Sp, Dp],
// decay, beta [B, H, Sp], kq [B, G] (decoding), coef [B, H, Sp / 16, COEF].
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
  float *q, *k, *v, *decay, *beta, *kq;
  int S, Sp, G, H, D, Dp, V, Vp, taps, has_past, nslots;
};

constexpr int CHUNK = 16;              // tokens per block of the preparation and per step of the scan
constexpr int P_PITCH = CHUNK + 4;     // row pitch of the o-from-u coefficients (conflict-free 16-byte reads of eight rows)
constexpr int COEF = CHUNK * P_PITCH + 2 * CHUNK;    // R_ij (q_i.k_j) for j <= i, then G_i, then R_last,i

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
  extern __shared__ float sqk[];         // [rows][2 Dp]; rows: CHUNK, or 4 when decoding
  const int s0 = blockIdx.x * CHUNK, b = blockIdx.z, tid = threadIdx.x, unit = blockIdx.y;
  const int len = p.lens ? p.lens[b] : p.S;
  if (s0 >= len) return;
  const int n = min(CHUNK, len - s0), nr = p.Sp == 1 ? 1 : CHUNK;      // rows n .. nr - 1 become tokens that change nothing
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
    for (int i = tid; i < (nr - n) * p.Vp; i += 128) vo[n * p.Vp + i] = 0.f;
    if (tid < nr) {
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
  const int rows = (nr + 3) / 4 * 4;
  if (p.D < Dp || n < rows)              // the tails of the rows, and rows without a token
    for (int i = tid; i < rows * W; i += 128)
      if (i / W >= n || i % Dp >= p.D) sqk[i] = 0.f;
  for (int d = tid; d < p.D; d += 128) {
    conv_channel<T, TAPS>(p, x0, hist, past, C, g * p.D + d, s0, n, [&](int i, float y) { sqk[i * W + d] = y; });
    conv_channel<T, TAPS>(p, x0, hist, past, C, (p.G + g) * p.D + d, s0, n, [&](int i, float y) { sqk[i * W + Dp + d] = y; });
  }
  __syncthreads();
  // one warp per four tokens: squares of their k (0-3) and q (4-7) and, for decoding, q_0.k_0 (8); reduced so that lanes 2 x and
  // 2 x + 1 hold sum x
  const int blk = tid >> 5, lane = tid & 31;
  if (blk * 4 >= nr) return;
  const float* base = sqk + blk * 4 * W;
  float pr[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) pr[i] = 0.f;
  for (int d = lane; d < Dp; d += 32) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float q = base[i * W + d], k = base[i * W + Dp + d];
      pr[i] = fmaf(k, k, pr[i]);
      pr[4 + i] = fmaf(q, q, pr[4 + i]);
      if (i == 0) pr[8] = fmaf(q, k, pr[8]);
    }
  }
#pragma unroll
  for (int m = 8; m > 0; m >>= 1) {      // m sums stay with each half of the lanes that share 2 m
    const bool up = lane & (2 * m);
#pragma unroll
    for (int i = 0; i < m; ++i) {
      const float send = up ? pr[i] : pr[i + m], keep = up ? pr[i + m] : pr[i];
      pr[i] = keep + __shfl_xor_sync(0xffffffffu, send, 2 * m);
    }
  }
  const float sum = pr[0] + __shfl_xor_sync(0xffffffffu, pr[0], 1);
  float r = 1.f / sqrtf(sum + 1e-6f);    // 1 / |k_i|, or 1 / (|q_i| sqrt(D))
  if (lane >= 8) r = r / sqrtf(float(p.D));
  float rk[4], rq[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    rk[i] = __shfl_sync(0xffffffffu, r, 2 * i);
    rq[i] = __shfl_sync(0xffffffffu, r, 8 + 2 * i);
  }
  const long long row0 = ((long long)b * p.G + g) * p.Sp + s0 + blk * 4;
  for (int d = lane; d < Dp; d += 32)
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (blk * 4 + i < nr) {
        p.q[(row0 + i) * Dp + d] = base[i * W + d] * rq[i];
        p.k[(row0 + i) * Dp + d] = base[i * W + Dp + d] * rk[i];
      }
  if (p.Sp == 1 && lane == 16) p.kq[(long long)b * p.G + g] = sum * rq[0] * rk[0];
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
// the part of 16 tokens' recurrence that does not need the state: w, y (over v) and the coefficients of o
// ------------------------------------------------------------------------------------------------
struct DeltaWyArgs {
  const float *q, *k, *decay, *beta;
  float *v, *w, *coef;
  const int* lens;
  int S, Sp, G, H, Dp, Vp;
};

__global__ void __launch_bounds__(128) delta_wy_kernel(const DeltaWyArgs p) {
  tfb::pdl_sync();
  extern __shared__ __align__(16) float ws[];
  __shared__ __align__(16) float sA[CHUNK][CHUNK];       // beta_i R_ij (k_i.k_j), j < i
  __shared__ float sd[CHUNK], sb[CHUNK], sg[CHUNK];      // decay, beta, G
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, g = h / (p.H / p.G);
  const int Dp = p.Dp, KP = Dp + 4;
  if (c * CHUNK >= (p.lens ? p.lens[b] : p.S)) return;
  float* sK = ws;
  float* sQ = ws + CHUNK * KP;
  const float4* kb = reinterpret_cast<const float4*>(p.k + (((long long)b * p.G + g) * p.Sp + c * CHUNK) * Dp);
  const float4* qb = reinterpret_cast<const float4*>(p.q + (((long long)b * p.G + g) * p.Sp + c * CHUNK) * Dp);
  for (int i = tid; i < CHUNK * Dp / 4; i += 128) {
    const int r = i / (Dp / 4), d = i % (Dp / 4) * 4;
    *reinterpret_cast<float4*>(sK + r * KP + d) = kb[i];
    *reinterpret_cast<float4*>(sQ + r * KP + d) = qb[i];
  }
  const long long hrow = ((long long)b * p.H + h) * p.Sp + c * CHUNK;
  if (tid < CHUNK) {
    sd[tid] = p.decay[hrow + tid];
    sb[tid] = p.beta[hrow + tid];
  }
  __syncthreads();
  if (tid < CHUNK) {
    float x = 1.f;
    for (int i = 0; i <= tid; ++i) x *= sd[i];
    sg[tid] = x;
  }
  float* coef = p.coef + (((long long)b * p.H + h) * (p.Sp / CHUNK) + c) * COEF;
  const int i = tid >> 3, j0 = tid & 7;
  float kk[2] = {0.f, 0.f}, qk[2] = {0.f, 0.f};
  for (int d = 0; d < Dp; d += 4) {
    const float4 ki = *reinterpret_cast<const float4*>(sK + i * KP + d), qi = *reinterpret_cast<const float4*>(sQ + i * KP + d);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float4 kj = *reinterpret_cast<const float4*>(sK + (j0 + 8 * e) * KP + d);
      kk[e] = fmaf(ki.x, kj.x, fmaf(ki.y, kj.y, fmaf(ki.z, kj.z, fmaf(ki.w, kj.w, kk[e]))));
      qk[e] = fmaf(qi.x, kj.x, fmaf(qi.y, kj.y, fmaf(qi.z, kj.z, fmaf(qi.w, kj.w, qk[e]))));
    }
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int j = j0 + 8 * e;
    float R = 1.f;
    for (int l = j + 1; l <= i; ++l) R *= sd[l];
    sA[i][j] = j < i ? sb[i] * R * kk[e] : 0.f;
    coef[i * P_PITCH + j] = j <= i ? R * qk[e] : 0.f;
    if (i == CHUNK - 1) coef[CHUNK * P_PITCH + CHUNK + j] = R;
  }
  __syncthreads();
  if (tid < CHUNK) coef[CHUNK * P_PITCH + tid] = sg[tid];
  else if (tid < 2 * CHUNK)
    for (int e = CHUNK; e < P_PITCH; ++e) coef[(tid - CHUNK) * P_PITCH + e] = 0.f;
  // forward substitution, one column per thread
  for (int col = tid; col < Dp + p.Vp; col += 128) {
    const bool is_k = col < Dp;
    float* vp = p.v + hrow * p.Vp + (col - Dp);
    float x[CHUNK];
#pragma unroll
    for (int r = 0; r < CHUNK; ++r) x[r] = is_k ? sb[r] * sg[r] * sK[r * KP + col] : sb[r] * vp[(long long)r * p.Vp];
#pragma unroll
    for (int r = 1; r < CHUNK; ++r) {
#pragma unroll
      for (int q = 0; q < (r + 3) / 4; ++q) {
        const float4 a = *reinterpret_cast<const float4*>(&sA[r][4 * q]);      // zeros from the diagonal on
        x[r] = fmaf(-a.x, x[4 * q], x[r]);
        if (4 * q + 1 < r) x[r] = fmaf(-a.y, x[4 * q + 1], x[r]);
        if (4 * q + 2 < r) x[r] = fmaf(-a.z, x[4 * q + 2], x[r]);
        if (4 * q + 3 < r) x[r] = fmaf(-a.w, x[4 * q + 3], x[r]);
      }
    }
    float* out = is_k ? p.w + hrow * Dp + col : vp;
    const int pitch = is_k ? Dp : p.Vp;
#pragma unroll
    for (int r = 0; r < CHUNK; ++r) out[(long long)r * pitch] = x[r];
  }
}

// ------------------------------------------------------------------------------------------------
// scan over a prompt
// ------------------------------------------------------------------------------------------------
struct DeltaScanArgs {
  const float *q, *k, *w, *y, *coef;
  float* o;               // [B*S, H, V]
  float* state;           // [slots, H, D, V]
  const int* state_slots; // [B]
  const int* lens;        // [B] or null
  int S, Sp, G, H, D, V, Vp, has_past, nslots;
  int* status;
};

typedef unsigned long long u64;
__device__ __forceinline__ u64 fma2(u64 a, u64 b, u64 c) {
  u64 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ u64 mul2(u64 a, u64 b) {
  u64 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ u64 pack2(float lo, float hi) {
  u64 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 unpack2(u64 v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}

// EPT: entries of one column per thread (a multiple of 4); TPC >= 8: threads per column group; CPT: columns per group;
// Dp = EPT TPC.  The products of token s ^ (t & 7) of a half chunk sit in register slot s of thread t, so that each round of the
// reduction adds a partner's upper slots to this thread's lower ones and thread t ends up with token t & 7.
template <int EPT, int TPC, int CPT>
__global__ void __launch_bounds__(128) delta_scan_kernel(const DeltaScanArgs p) {
  tfb::pdl_sync();
  extern __shared__ __align__(128) float sm[];
  constexpr int Dp = EPT * TPC, CPW = 32 / TPC * CPT;
  static_assert(TPC >= 8 && EPT % 4 == 0 && CHUNK == 16, "tile shape");
  const int tid = threadIdx.x, lane = tid & 31, cols = (blockDim.x >> 5) * CPW;
  const int h = blockIdx.y, b = blockIdx.z, g = h / (p.H / p.G), col0 = blockIdx.x * cols;
  const int t = lane % TPC, t8 = t & 7, cl = (tid >> 5) * CPW + lane / TPC * CPT;   // first column of the group, within the block
  const int len = p.lens ? p.lens[b] : p.S;
  const int stage_f = 3 * CHUNK * Dp + CHUNK * cols + COEF;
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
  const float* wb = p.w + ((long long)b * p.H + h) * p.Sp * Dp;
  const float* yb = p.y + ((long long)b * p.H + h) * p.Sp * p.Vp + col0;
  const float* cb = p.coef + ((long long)b * p.H + h) * (p.Sp / CHUNK) * COEF;
  const int nchunk = (len + CHUNK - 1) / CHUNK, nc = min(cols, p.Vp - col0);
  auto issue = [&](int c) {              // warp 0: the rows of chunk c
    if (c >= nchunk || tid >= 32) return;
    float* base = sm + (c & 1) * stage_f;
    const uint32_t br = bar + (c & 1) * 8;
    if (lane == 0) mbar_expect_tx(br, uint32_t(CHUNK * (3 * Dp + nc) + COEF) * 4);
    __syncwarp();
    if (lane == 0) bulk_load(smem_u32(base), wb + (long long)c * CHUNK * Dp, CHUNK * Dp * 4, br);
    if (lane == 1) bulk_load(smem_u32(base + CHUNK * Dp), qb + (long long)c * CHUNK * Dp, CHUNK * Dp * 4, br);
    if (lane == 2) bulk_load(smem_u32(base + 2 * CHUNK * Dp), kb + (long long)c * CHUNK * Dp, CHUNK * Dp * 4, br);
    if (lane == 3) bulk_load(smem_u32(base + 3 * CHUNK * Dp + CHUNK * cols), cb + (long long)c * COEF, COEF * 4, br);
    if (lane >= 16)
      bulk_load(smem_u32(base + 3 * CHUNK * Dp + (lane - 16) * cols), yb + (long long)(c * CHUNK + lane - 16) * p.Vp, nc * 4, br);
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

  const long long ostep = (long long)p.H * p.V;
  float* orow = p.o + ((long long)b * p.S * p.H + h) * p.V + col0 + cl;
  for (int c = 0; c < nchunk; ++c) {
    if (!mbar_wait_warp(bar + (c & 1) * 8, (c >> 1) & 1, abort_flag, p.status, ST_TIMEOUT_FULL)) break;
    const float* base = sm + (c & 1) * stage_f;
    const float* sy = base + 3 * CHUNK * Dp;
    const float* sc = sy + CHUNK * cols;
    float um[2][CPT], oq[2][CPT];        // u, and S^T q, of tokens t8 and t8 + 8
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      float val[8][2 * CPT];             // [slot][2 column + (w: 0, q: 1)]
#pragma unroll
      for (int s = 0; s < 8; ++s) {
        const ulonglong2* sw = reinterpret_cast<const ulonglong2*>(base + (half * 8 + (s ^ t8)) * Dp) + t;
        const ulonglong2* sq = sw + CHUNK * Dp / 4;
        u64 a[EPT / 2];
#pragma unroll
        for (int y = 0; y < 2; ++y) {
#pragma unroll
          for (int e = 0; e < EPT / 4; ++e) {
            const ulonglong2 r = y ? sq[e * TPC] : sw[e * TPC];
            a[2 * e] = r.x;
            a[2 * e + 1] = r.y;
          }
#pragma unroll
          for (int x = 0; x < CPT; ++x) {
            u64 d = mul2(st[x][0], a[0]);
#pragma unroll
            for (int e = 1; e < EPT / 2; ++e) d = fma2(st[x][e], a[e], d);
            const float2 f = unpack2(d);
            val[s][2 * x + y] = f.x + f.y;
          }
        }
      }
#pragma unroll
      for (int o = TPC >> 1; o >= 8; o >>= 1)
#pragma unroll
        for (int s = 0; s < 8; ++s)
#pragma unroll
          for (int y = 0; y < 2 * CPT; ++y) val[s][y] += __shfl_xor_sync(0xffffffffu, val[s][y], o);
#pragma unroll
      for (int o = 4; o > 0; o >>= 1)
#pragma unroll
        for (int s = 0; s < o; ++s)
#pragma unroll
          for (int y = 0; y < 2 * CPT; ++y) val[s][y] += __shfl_xor_sync(0xffffffffu, val[s + o][y], o);
#pragma unroll
      for (int x = 0; x < CPT; ++x) {
        um[half][x] = sy[(half * 8 + t8) * cols + cl + x] - val[0][2 * x];
        oq[half][x] = val[0][2 * x + 1];
      }
    }
    // every thread gets the 16 u of its columns
    float u[CPT][CHUNK];
#pragma unroll
    for (int x = 0; x < CPT; ++x)
#pragma unroll
      for (int j = 0; j < CHUNK; ++j) u[x][j] = __shfl_sync(0xffffffffu, um[j >> 3][x], (lane & ~(TPC - 1)) + (j & 7));
    const float* sG = sc + CHUNK * P_PITCH;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int row = half * 8 + t8, tok = c * CHUNK + row;
      const float4* pr = reinterpret_cast<const float4*>(sc + row * P_PITCH);
      const float gi = sG[row];
      float ov[CPT];
#pragma unroll
      for (int x = 0; x < CPT; ++x) ov[x] = gi * oq[half][x];
#pragma unroll
      for (int j = 0; j < 2 * (half + 1); ++j) {          // tokens 0-7 have no coefficients past the first eight
        const float4 f = pr[j];
#pragma unroll
        for (int x = 0; x < CPT; ++x)
          ov[x] = fmaf(f.w, u[x][4 * j + 3], fmaf(f.z, u[x][4 * j + 2], fmaf(f.y, u[x][4 * j + 1], fmaf(f.x, u[x][4 * j], ov[x]))));
      }
      if (t < 8 && tok < len) {
#pragma unroll
        for (int x = 0; x < CPT; ++x)
          if (col0 + cl + x < p.V) orow[(long long)tok * ostep + x] = ov[x];
      }
    }
    const u64 gl = pack2(sG[CHUNK - 1], sG[CHUNK - 1]);
#pragma unroll
    for (int x = 0; x < CPT; ++x)
#pragma unroll
      for (int e = 0; e < EPT / 2; ++e) st[x][e] = mul2(st[x][e], gl);
    const float4* sR = reinterpret_cast<const float4*>(sG + CHUNK);
#pragma unroll
    for (int j = 0; j < CHUNK; ++j) {
      const float4 R4 = sR[j >> 2];
      const float R = (j & 3) == 0 ? R4.x : (j & 3) == 1 ? R4.y : (j & 3) == 2 ? R4.z : R4.w;
      const ulonglong2* sk = reinterpret_cast<const ulonglong2*>(base + (2 * CHUNK + j) * Dp) + t;
      u64 a[EPT / 2];
#pragma unroll
      for (int e = 0; e < EPT / 4; ++e) {
        const ulonglong2 r = sk[e * TPC];
        a[2 * e] = r.x;
        a[2 * e + 1] = r.y;
      }
#pragma unroll
      for (int x = 0; x < CPT; ++x) {
        const float f = u[x][j] * R;
        const u64 ff = pack2(f, f);
#pragma unroll
        for (int e = 0; e < EPT / 2; ++e) st[x][e] = fma2(a[e], ff, st[x][e]);
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
  auto bytes = [](int w) { return (2 * (3 * CHUNK * EPT * TPC + CHUNK * w * CPW + COEF) + 8) * int(sizeof(float)); };
  if (nw < 1 || nw > 4 || (nw * CPW) % 4) return TFB_ERR_ARG;      // rows of y are copied in 16-byte pieces
  static DeviceOnce once;
  auto kern = delta_scan_kernel<EPT, TPC, CPT>;
  if (int e = ensure_dyn_smem(once, kern, bytes(4))) return e;
  const int cols = nw * CPW;
  launch_k(kern, dim3((p.V + cols - 1) / cols, p.H, B), nw * 32, bytes(nw), st, p);
  return int(cudaGetLastError());
}

template <int EPT, int TPC>
static int launch_scan(const DeltaScanArgs& p, int B, int tile, cudaStream_t st) {
  // Wide groups (four columns) read w, q and k from shared memory a quarter as often; narrow ones spread few sequences over more
  // warps.
  constexpr int GPW = 32 / TPC;
  auto warps = [&](int cpt) { return (long long)((p.V + GPW * cpt - 1) / (GPW * cpt)) * p.H * B; };
  int cpt = warps(4) >= 3ll * sm_count() ? 4 : warps(2) >= sm_count() ? 2 : 1, nw = 4;
  while (nw > 1 && nw / 2 * GPW * cpt >= 4 && (nw * GPW * cpt > (p.V + 3) / 4 * 4 || (warps(cpt) + nw - 1) / nw < 4 * sm_count() / 5)) nw >>= 1;
  if (tile > 0) {
    cpt = tile >> 4;
    nw = tile & 15;
  }
  switch (cpt) {
    case 1: return launch_scan_tile<EPT, TPC, 1>(p, B, nw, st);
    case 2: return launch_scan_tile<EPT, TPC, 2>(p, B, nw, st);
    case 4: return launch_scan_tile<EPT, TPC, 4>(p, B, nw, st);
    default: return TFB_ERR_ARG;
  }
}

// ------------------------------------------------------------------------------------------------
// gated norm of the head outputs:  o / rms(o) * w * silu(gate)
// ------------------------------------------------------------------------------------------------
template <class T, int VEC>
__global__ void __launch_bounds__(256) gated_norm_kernel(const float* __restrict__ o, const T* __restrict__ gate, long long ldg,
                                                         const T* __restrict__ w, T* __restrict__ out, long long ldo, int rows, int H, int V,
                                                         float eps) {
  tfb::pdl_sync();
  const int lane = threadIdx.x & 31;
  const long long nwarps = (long long)gridDim.x * (blockDim.x >> 5), n = (long long)rows * H;
  for (long long i = blockIdx.x * (long long)(blockDim.x >> 5) + (threadIdx.x >> 5); i < n; i += nwarps) {
    const long long r = i / H;
    const int h = int(i % H);
    const float* src = o + i * V;
    const T* gt = gate + r * ldg + h * V;
    T* dst = out + r * ldo + h * V;
    float x0[VEC], g0[VEC], x[VEC], g[VEC], wv[VEC];
    float ss = 0.f;
    for (int j = lane * VEC; j < V; j += 32 * VEC) {
      load_n<VEC>(src + j, x);
      if (j == lane * VEC) {
        load_n<VEC>(gt + j, g0);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x0[e] = x[e];
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss = fmaf(x[e], x[e], ss);
    }
    const float rs = 1.f / sqrtf(warp_add(ss) / V + eps);
    for (int j = lane * VEC; j < V; j += 32 * VEC) {
      load_n<VEC>(w + j, wv);
      if (j == lane * VEC) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) { x[e] = x0[e]; g[e] = g0[e]; }
      } else {
        load_n<VEC>(src + j, x);
        load_n<VEC>(gt + j, g);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] = x[e] * rs * wv[e] * silu_exact(g[e]);
      store_n<VEC>(dst + j, x);
    }
  }
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

// Convolution, activation, unit lengths, gates and (Sp > 1) w, y and the coefficients of B sequences with S rows each, lens[b] of them
// real.  has_past: the history in conv_state belongs to these sequences (otherwise they start here and see zeros).
TFB_API int tfb_delta_prep(const void* proj, long long ld, const void* conv_w, void* conv_state, const int* state_slots, int nslots,
                           const void* A_log, const void* dt_bias, const int* lens, float* q, float* k, float* v, float* decay, float* beta,
                           float* kq, float* w, float* coef, int B, int S, int Sp, int G, int H, int D, int V, int taps, int has_past, int f32,
                           void* stream) {
  using namespace tfb;
  const int Dp = tfb_delta_padded_dim(D);
  if (B <= 0 || B > 65535 || S <= 0 || G <= 0 || H % G || G + H > 65535 || D <= 0 || V <= 0 || taps < 1) return TFB_ERR_ARG;
  if (Sp != 1 && (Sp != (S + CHUNK - 1) / CHUNK * CHUNK || !coef || !w)) return TFB_ERR_ARG;
  if (Sp == 1 && S != 1) return TFB_ERR_ARG;
  if (!Dp) return TFB_ERR_LIMIT;
  DeltaPrepArgs p{proj, ld, conv_w, conv_state, state_slots, A_log, dt_bias, lens, q, k, v, decay, beta, kq,
                  S, Sp, G, H, D, Dp, V, (V + 3) / 4 * 4, taps, has_past, nslots};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 grid((Sp + CHUNK - 1) / CHUNK, G + H, B);
  const int smem = (Sp == 1 ? 4 : CHUNK) * 2 * Dp * int(sizeof(float));     // at most 64 KB
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
  if (Sp > 1) {
    static DeviceOnce once;
    if (int e = ensure_dyn_smem(once, delta_wy_kernel, 2 * CHUNK * (512 + 4) * int(sizeof(float)))) return e;
    DeltaWyArgs a{q, k, decay, beta, v, w, coef, lens, S, Sp, G, H, Dp, (V + 3) / 4 * 4};
    launch_k(delta_wy_kernel, dim3(Sp / CHUNK, H, B), 128, 2 * CHUNK * (Dp + 4) * int(sizeof(float)), st, a);
  }
  return int(cudaGetLastError());
}

// The recurrence over the prepared rows (Sp > 1); o [B*S, H, V] fp32.
// tile 0: the launch shape is chosen from the sizes; 16 CPT + warps per block: that shape (CPT 1, 2 or 4; up to 4 warps).
TFB_API int tfb_delta_scan(const float* q, const float* k, const float* w, const float* y, const float* coef, float* o, float* state, const int* state_slots,
                           int nslots, const int* lens, int B, int S, int G, int H, int D, int V, int has_past, int tile, int* status, void* stream) {
  using namespace tfb;
  if (B <= 0 || B > 65535 || S <= 0 || G <= 0 || H % G || H > 65535 || D <= 0 || V <= 0) return TFB_ERR_ARG;
  DeltaScanArgs p{q, k, w, y, coef, o, state, state_slots, lens, S, (S + CHUNK - 1) / CHUNK * CHUNK, G, H, D, V, (V + 3) / 4 * 4, has_past, nslots, status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  switch (tfb_delta_padded_dim(D)) {
    case 32: return launch_scan<4, 8>(p, B, tile, st);
    case 64: return launch_scan<8, 8>(p, B, tile, st);
    case 128: return launch_scan<16, 8>(p, B, tile, st);
    case 256: return launch_scan<16, 16>(p, B, tile, st);
    case 512: return launch_scan<16, 32>(p, B, tile, st);
    default: return TFB_ERR_LIMIT;
  }
}

TFB_API int tfb_gated_norm(const float* o, const void* gate, long long ldg, const void* w, void* out, long long ldo, int rows, int H, int V,
                           float eps, int f32, void* stream) {
  using namespace tfb;
  if (rows <= 0 || H <= 0 || V <= 0) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const long long blocks = ((long long)rows * H + 7) / 8;
  const int grid = int(blocks < 148ll * 32 ? blocks : 148ll * 32);
  auto al = [](const void* x, int n) { return (reinterpret_cast<uintptr_t>(x) & (n - 1)) == 0; };
  const int es = f32 ? 4 : 2;
  const bool v4 = V % 4 == 0 && ldg % 4 == 0 && ldo % 4 == 0 && al(o, 16) && al(gate, 4 * es) && al(w, 4 * es) && al(out, 4 * es);
#define TFB_GN(T, VEC) launch_k(gated_norm_kernel<T, VEC>, grid, 256, 0, st, o, static_cast<const T*>(gate), ldg, static_cast<const T*>(w), \
                                static_cast<T*>(out), ldo, rows, H, V, eps)
  if (f32) { if (v4) TFB_GN(float, 4); else TFB_GN(float, 1); }
  else { if (v4) TFB_GN(bf16, 4); else TFB_GN(bf16, 1); }
#undef TFB_GN
  return int(cudaGetLastError());
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
