// Gated delta rule (linear attention with a per-head state matrix) for prompts and for decoding.
//
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q            per head, S is [D, V] in fp32
//
// Three kernels:
//   delta_prep   one block per token row: causal convolution of q, k and v over time (per channel, with the last inputs of
//                the previous step as history), silu, unit length of q and k per head, the decay g and the step size beta.
//                Everything it hands on is fp32.
//   delta_scan   prompts.  The columns of S are independent recurrences that share k and q, so a group of TPC threads
//                owns one column (D / TPC entries each, in registers as packed fp32 pairs) and walks over the tokens; k,
//                q, v and the gates of the next tokens travel to shared memory (cp.async) while the current ones are used.
//                S^T k and S^T q are taken from the same old state (o = g S^T q + (k.q) u), so a token has one reduction
//                on its critical path instead of two.  The state never leaves the registers between tokens, and the
//                arithmetic is fp32 FMA throughout: how a prompt is cut into portions changes nothing.
//   delta_step   one token per sequence: one block per (sequence, head) streams the state through registers once (read,
//                two products, rank-one update, write) and applies the gated norm of the head's output.
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
  float *q, *k, *v;       // [B*S, G, D], [B*S, G, D], [B*S, H, V]
  float *kq;              // [B*S, G]: k . q
  float *decay, *beta;    // [B*S, H]
  int S, G, H, D, V, taps, has_past, nslots;
};

template <class T>
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaPrepArgs p) {
  tfb::pdl_sync();
  extern __shared__ float sqk[];                      // 2 G D activated q and k channels
  const int s = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int len = p.lens ? p.lens[b] : p.S;
  if (s >= len) return;
  const long long r = (long long)b * p.S + s;
  const int nqk = 2 * p.G * p.D, C = nqk + p.H * p.V, taps = p.taps;
  const T* x = static_cast<const T*>(p.proj) + r * p.ld;
  const T* cw = static_cast<const T*>(p.conv_w);
  int slot = p.state_slots ? p.state_slots[b] : -1;
  TFB_BOUNDS(slot < p.nslots, 71, slot, p.nslots);
  if (slot >= p.nslots) slot = -1;
  T* hist = (slot >= 0 && taps > 1) ? static_cast<T*>(p.conv_state) + (long long)slot * (taps - 1) * C : nullptr;
  const bool past = hist && p.has_past;
  for (int c = tid; c < C; c += blockDim.x) {
    const float cur = to_f(x[c]);
    float y = 0.f;
    for (int j = 0; j < taps - 1; ++j) {
      const int t = s - (taps - 1) + j;               // token index within this call; negative: history
      float in = 0.f;
      if (t >= 0) in = to_f(x[(long long)(t - s) * p.ld + c]);
      else if (past) in = to_f(hist[(long long)(taps - 1 + t) * C + c]);
      y = fmaf(to_f(cw[(long long)c * taps + j]), in, y);
    }
    y = fmaf(to_f(cw[(long long)c * taps + taps - 1]), cur, y);
    y = silu_exact(y);
    if (c < nqk) sqk[c] = y;
    else p.v[r * p.H * p.V + (c - nqk)] = y;
    if (p.S == 1 && hist) {                           // decoding: this thread alone uses channel c, so the window moves in place
      for (int j = 0; j < taps - 2; ++j) hist[(long long)j * C + c] = past ? hist[(long long)(j + 1) * C + c] : from_f<T>(0.f);
      hist[(long long)(taps - 2) * C + c] = x[c];
    }
  }
  const T* gb = x + C + p.H * p.V;
  for (int h = tid; h < p.H; h += blockDim.x) {
    const float bz = to_f(gb[h]);
    const float z = to_f(gb[p.H + h]) + to_f(static_cast<const T*>(p.dt_bias)[h]);
    const float sp = z > 20.f ? z : log1pf(expf(z));
    p.beta[r * p.H + h] = 1.f / (1.f + expf(-bz));
    p.decay[r * p.H + h] = expf(-expf(to_f(static_cast<const T*>(p.A_log)[h])) * sp);
  }
  __syncthreads();
  const int warp = tid >> 5, lane = tid & 31;
  for (int g = warp; g < p.G; g += blockDim.x >> 5) {
    const float* sq = sqk + g * p.D;
    const float* sk = sqk + (p.G + g) * p.D;
    float qq = 0.f, kk = 0.f, qk = 0.f;
    for (int d = lane; d < p.D; d += 32) {
      qq = fmaf(sq[d], sq[d], qq);
      kk = fmaf(sk[d], sk[d], kk);
      qk = fmaf(sq[d], sk[d], qk);
    }
    qq = warp_add(qq);
    kk = warp_add(kk);
    qk = warp_add(qk);
    const float rq = 1.f / sqrtf(qq + 1e-6f) / sqrtf(float(p.D)), rk = 1.f / sqrtf(kk + 1e-6f);
    float* oq = p.q + (r * p.G + g) * p.D;
    float* ok = p.k + (r * p.G + g) * p.D;
    for (int d = lane; d < p.D; d += 32) {
      oq[d] = sq[d] * rq;
      ok[d] = sk[d] * rk;
    }
    if (lane == 0) p.kq[r * p.G + g] = qk * rq * rk;
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
// scan over a prompt
// ------------------------------------------------------------------------------------------------
struct DeltaScanArgs {
  const float *q, *k, *v, *kq, *decay, *beta;
  float* o;               // [B*S, H, V]
  float* state;           // [slots, H, D, V]
  const int* state_slots; // [B]
  const int* lens;        // [B] or null
  int S, G, H, D, V, has_past, nslots;
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
__device__ __forceinline__ void cp_async_bytes16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_bytes4(uint32_t dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory");
}

constexpr int SCAN_CHUNK = 16;   // tokens per shared-memory stage

// EPT: entries of one column per thread (a multiple of 4); TPC: threads per column; D <= EPT * TPC.
// Shared memory per stage: k, q [CHUNK][Dp] (Dp = EPT * TPC, the tail is zero), v [CHUNK][cols], and 3 scalars per token.
template <int EPT, int TPC>
__global__ void delta_scan_kernel(const DeltaScanArgs p) {
  tfb::pdl_sync();
  extern __shared__ __align__(16) float sm[];
  constexpr int Dp = EPT * TPC, CPW = 32 / TPC;
  const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31;
  const int cols = (nt >> 5) * CPW;
  const int h = blockIdx.y, b = blockIdx.z, g = h / (p.H / p.G), col0 = blockIdx.x * cols;
  const int cl = (tid >> 5) * CPW + lane / TPC, t = lane % TPC, col = col0 + cl;
  const bool live = col < p.V;
  const int len = p.lens ? p.lens[b] : p.S;
  const long long r0 = (long long)b * p.S;
  const int stage_f = 2 * SCAN_CHUNK * Dp + SCAN_CHUNK * cols + 4 * SCAN_CHUNK;
  const bool vec_d = (p.D & 3) == 0, vec_v = (p.V & 3) == 0 && (cols & 3) == 0;
  const int cshift = 31 - __clz(cols);      // cols is a power of two

  for (int i = tid; i < 2 * stage_f; i += nt) sm[i] = 0.f;      // tails of k and q stay zero
  int slot = p.state_slots ? p.state_slots[b] : -1;
  TFB_BOUNDS(slot < p.nslots, 72, slot, p.nslots);
  if (slot >= p.nslots) slot = -1;
  float* S0 = slot >= 0 ? p.state + ((long long)slot * p.H + h) * p.D * p.V : nullptr;
  // entry d of the column sits with thread (d / 4) % TPC, register (d / 4) / TPC * 4 + d % 4
  u64 st[EPT / 2];
#pragma unroll
  for (int i = 0; i < EPT / 4; ++i) {
    float f[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = (i * TPC + t) * 4 + e;
      f[e] = (S0 && p.has_past && live && d < p.D) ? S0[(long long)d * p.V + col] : 0.f;
    }
    st[2 * i] = pack2(f[0], f[1]);
    st[2 * i + 1] = pack2(f[2], f[3]);
  }
  __syncthreads();

  auto issue = [&](int c) {
    const int s0 = c * SCAN_CHUNK, n = min(SCAN_CHUNK, len - s0);
    float* base = sm + (c & 1) * stage_f;
    if (n > 0) {
      constexpr int QV = Dp / 4;                                 // index arithmetic in powers of two
      for (int i = tid; i < 2 * SCAN_CHUNK * QV; i += nt) {
        const int w = i / (SCAN_CHUNK * QV), tk = (i / QV) % SCAN_CHUNK, d = (i % QV) * 4;
        if (tk >= n || d >= p.D) continue;
        const float* src = (w ? p.q : p.k) + ((r0 + s0 + tk) * p.G + g) * p.D + d;
        const uint32_t dst = smem_u32(base + (w * SCAN_CHUNK + tk) * Dp + d);
        if (vec_d) cp_async_bytes16(dst, src);
        else
          for (int e = 0; e < min(4, p.D - d); ++e) cp_async_bytes4(dst + 4 * e, src + e);
      }
      float* sv = base + 2 * SCAN_CHUNK * Dp;
      const int vs = vec_v ? cshift - 2 : cshift;
      for (int i = tid; i < (SCAN_CHUNK << vs); i += nt) {
        const int tk = i >> vs, j = (i & ((1 << vs) - 1)) << (cshift - vs);
        if (tk >= n || col0 + j >= p.V) continue;
        const float* src = p.v + ((r0 + s0 + tk) * p.H + h) * p.V + col0 + j;
        if (vec_v) cp_async_bytes16(smem_u32(sv + tk * cols + j), src);
        else cp_async_bytes4(smem_u32(sv + tk * cols + j), src);
      }
      float* sg = sv + SCAN_CHUNK * cols;
      for (int i = tid; i < 4 * SCAN_CHUNK; i += nt) {
        const int tk = i >> 2, w = i & 3;
        if (tk >= n || w == 3) continue;
        const float* src = w == 0 ? p.decay + (r0 + s0 + tk) * p.H + h : w == 1 ? p.beta + (r0 + s0 + tk) * p.H + h : p.kq + (r0 + s0 + tk) * p.G + g;
        cp_async_bytes4(smem_u32(sg + tk * 4 + w), src);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  const int nchunk = (len + SCAN_CHUNK - 1) / SCAN_CHUNK;
  issue(0);
  for (int c = 0; c < nchunk; ++c) {
    issue(c + 1);
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const float* base = sm + (c & 1) * stage_f;
    const float* sv = base + 2 * SCAN_CHUNK * Dp;
    const float* sg = sv + SCAN_CHUNK * cols;
    const int n = min(SCAN_CHUNK, len - c * SCAN_CHUNK);
    float* orow = p.o + ((r0 + c * SCAN_CHUNK) * p.H + h) * p.V + col;
#pragma unroll 2
    for (int tk = 0; tk < n; ++tk) {
      const ulonglong2* sk = reinterpret_cast<const ulonglong2*>(base + tk * Dp) + t;
      const ulonglong2* sq = reinterpret_cast<const ulonglong2*>(base + (SCAN_CHUNK + tk) * Dp) + t;
      const float4 gs = *reinterpret_cast<const float4*>(sg + tk * 4);     // decay, beta, k.q
      const float v = sv[tk * cols + cl];
      u64 kk[EPT / 2];
      u64 dk0 = 0, dk1 = 0, dq0 = 0, dq1 = 0;
#pragma unroll
      for (int i = 0; i < EPT / 4; ++i) {
        const ulonglong2 a = sk[i * TPC], q = sq[i * TPC];
        kk[2 * i] = a.x;
        kk[2 * i + 1] = a.y;
        dk0 = fma2(st[2 * i], a.x, dk0);
        dk1 = fma2(st[2 * i + 1], a.y, dk1);
        dq0 = fma2(st[2 * i], q.x, dq0);
        dq1 = fma2(st[2 * i + 1], q.y, dq1);
      }
      const float2 ka = unpack2(dk0), kb = unpack2(dk1), qa = unpack2(dq0), qb = unpack2(dq1);
      float dk = (ka.x + ka.y) + (kb.x + kb.y), dq = (qa.x + qa.y) + (qb.x + qb.y);
#pragma unroll
      for (int o = TPC >> 1; o > 0; o >>= 1) {
        dk += __shfl_xor_sync(0xffffffffu, dk, o);
        dq += __shfl_xor_sync(0xffffffffu, dq, o);
      }
      const float u = gs.y * (v - gs.x * dk);
      const u64 uu = pack2(u, u), gg = pack2(gs.x, gs.x);
#pragma unroll
      for (int i = 0; i < EPT / 2; ++i) st[i] = fma2(kk[i], uu, mul2(st[i], gg));
      if (t == 0 && live) orow[(long long)tk * p.H * p.V] = fmaf(gs.x, dq, gs.z * u);
    }
    __syncthreads();
  }
  if (S0 && live) {
#pragma unroll
    for (int i = 0; i < EPT / 4; ++i) {
      const float2 a = unpack2(st[2 * i]), c = unpack2(st[2 * i + 1]);
      const float f[4] = {a.x, a.y, c.x, c.y};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = (i * TPC + t) * 4 + e;
        if (d < p.D) S0[(long long)d * p.V + col] = f[e];
      }
    }
  }
}

template <int EPT, int TPC>
static int launch_scan(const DeltaScanArgs& p, int B, cudaStream_t st) {
  // warps per block: few blocks leave SMs idle when there is one sequence, many small blocks fetch k and q more often
  int nw = 4;
  const int cpw = 32 / TPC;
  while (nw > 1 && (long long)((p.V + nw * cpw - 1) / (nw * cpw)) * p.H * B < sm_count()) nw >>= 1;
  const int cols = nw * cpw;
  const int smem = 2 * (2 * SCAN_CHUNK * EPT * TPC + SCAN_CHUNK * cols + 4 * SCAN_CHUNK) * int(sizeof(float));
  static DeviceOnce once;
  auto kern = delta_scan_kernel<EPT, TPC>;
  if (int e = ensure_dyn_smem(once, kern, 2 * (2 * SCAN_CHUNK * EPT * TPC + SCAN_CHUNK * 4 * cpw + 4 * SCAN_CHUNK) * int(sizeof(float)))) return e;
  launch_k(kern, dim3((p.V + cols - 1) / cols, p.H, B), nw * 32, smem, st, p);
  return int(cudaGetLastError());
}

// ------------------------------------------------------------------------------------------------
// gated norm of the head outputs:  o / rms(o) * w * silu(gate)
// ------------------------------------------------------------------------------------------------
template <class T>
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
    float ss = 0.f;
    for (int j = lane; j < V; j += 32) ss = fmaf(src[j], src[j], ss);
    const float rs = 1.f / sqrtf(warp_add(ss) / V + eps);
    for (int j = lane; j < V; j += 32)
      out[r * ldo + h * V + j] = from_f<T>(src[j] * rs * to_f(w[j]) * silu_exact(to_f(gate[r * ldg + h * V + j])));
  }
}

// ------------------------------------------------------------------------------------------------
// one token per sequence
// ------------------------------------------------------------------------------------------------
// 256 threads = 8 warps; warp w holds rows w, w + 8, ... (NR of them) of the state, lane l the columns 4 l .. 4 l + 3 of
// each 128-column part.  D <= 8 NR, V <= 128 CV, V % 4 == 0.
template <class T, int NR, int CV>
__global__ void __launch_bounds__(256) delta_step_kernel(const DeltaScanArgs p, const T* __restrict__ gate, long long ldg,
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
    sk[d] = d < p.D ? p.k[((long long)b * p.G + g) * p.D + d] : 0.f;
    sq[d] = d < p.D ? p.q[((long long)b * p.G + g) * p.D + d] : 0.f;
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
    const float u = bet * (p.v[((long long)b * p.H + h) * p.V + tid] - dec * dk);
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
static int launch_step(const DeltaScanArgs& p, int B, const void* gate, long long ldg, const void* w, void* out, long long ldo, float eps,
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

// Convolution, activation, unit lengths and gates of B sequences with S rows each (lens[b] of them real).  has_past: the
// history in conv_state belongs to these sequences (otherwise they start here and see zeros).
TFB_API int tfb_delta_prep(const void* proj, long long ld, const void* conv_w, void* conv_state, const int* state_slots, int nslots,
                           const void* A_log, const void* dt_bias, const int* lens, float* q, float* k, float* v, float* kq, float* decay,
                           float* beta, int B, int S, int G, int H, int D, int V, int taps, int has_past, int f32, void* stream) {
  using namespace tfb;
  if (B <= 0 || B > 65535 || S <= 0 || G <= 0 || H % G || D <= 0 || V <= 0 || taps < 1) return TFB_ERR_ARG;
  const int smem = 2 * G * D * int(sizeof(float));
  if (smem > 200 * 1024) return TFB_ERR_LIMIT;
  DeltaPrepArgs p{proj, ld, conv_w, conv_state, state_slots, A_log, dt_bias, lens, q, k, v, kq, decay, beta, S, G, H, D, V, taps, has_past, nslots};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  static DeviceOnce once16, once32;
  if (f32) {
    if (int e = ensure_dyn_smem(once32, delta_prep_kernel<float>, 200 * 1024)) return e;
    launch_k(delta_prep_kernel<float>, dim3(S, B), 256, smem, st, p);
  } else {
    if (int e = ensure_dyn_smem(once16, delta_prep_kernel<bf16>, 200 * 1024)) return e;
    launch_k(delta_prep_kernel<bf16>, dim3(S, B), 256, smem, st, p);
  }
  if (S > 1 && taps > 1 && state_slots) {
    const dim3 grid((2 * G * D + H * V + 255) / 256, B);
    if (f32) launch_k(conv_history_kernel<float>, grid, 256, 0, st, p);
    else launch_k(conv_history_kernel<bf16>, grid, 256, 0, st, p);
  }
  return int(cudaGetLastError());
}

// The recurrence over the prepared rows; o [B*S, H, V] fp32.
TFB_API int tfb_delta_scan(const float* q, const float* k, const float* v, const float* kq, const float* decay, const float* beta, float* o,
                           float* state, const int* state_slots, int nslots, const int* lens, int B, int S, int G, int H, int D, int V,
                           int has_past, void* stream) {
  using namespace tfb;
  if (B <= 0 || B > 65535 || S <= 0 || G <= 0 || H % G || H > 65535 || D <= 0 || V <= 0) return TFB_ERR_ARG;
  DeltaScanArgs p{q, k, v, kq, decay, beta, o, state, state_slots, lens, S, G, H, D, V, has_past, nslots};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (D <= 32) return launch_scan<8, 4>(p, B, st);
  if (D <= 64) return launch_scan<16, 4>(p, B, st);
  if (D <= 128) return launch_scan<32, 4>(p, B, st);
  if (D <= 256) return launch_scan<32, 8>(p, B, st);
  if (D <= 512) return launch_scan<32, 16>(p, B, st);
  return TFB_ERR_LIMIT;
}

TFB_API int tfb_gated_norm(const float* o, const void* gate, long long ldg, const void* w, void* out, long long ldo, int rows, int H, int V,
                           float eps, int f32, void* stream) {
  using namespace tfb;
  if (rows <= 0 || H <= 0 || V <= 0) return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const long long blocks = ((long long)rows * H + 7) / 8;
  const int grid = int(blocks < 148ll * 16 ? blocks : 148ll * 16);
  if (f32) launch_k(gated_norm_kernel<float>, grid, 256, 0, st, o, static_cast<const float*>(gate), ldg, static_cast<const float*>(w),
                    static_cast<float*>(out), ldo, rows, H, V, eps);
  else launch_k(gated_norm_kernel<bf16>, grid, 256, 0, st, o, static_cast<const bf16*>(gate), ldg, static_cast<const bf16*>(w),
                static_cast<bf16*>(out), ldo, rows, H, V, eps);
  return int(cudaGetLastError());
}

// One token for each of B sequences, gated norm included.  Returns TFB_ERR_LIMIT for head sizes it does not hold in
// registers (the caller then takes the scan with S = 1 and the norm kernel).
TFB_API int tfb_delta_step(const float* q, const float* k, const float* v, const float* kq, const float* decay, const float* beta, float* state,
                           const int* state_slots, int nslots, const void* gate, long long ldg, const void* w, void* out, long long ldo, int B,
                           int G, int H, int D, int V, int has_past, float eps, int f32, void* stream) {
  using namespace tfb;
  if (B <= 0 || B > 65535 || G <= 0 || H % G || D <= 0 || V <= 0 || !state_slots) return TFB_ERR_ARG;
  if ((V & 3) || V > 256 || D > 256 || (V > 128 && D > 128)) return TFB_ERR_LIMIT;
  DeltaScanArgs p{q, k, v, kq, decay, beta, nullptr, state, state_slots, nullptr, 1, G, H, D, V, has_past, nslots};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return f32 ? launch_step<float>(p, B, gate, ldg, w, out, ldo, eps, st) : launch_step<bf16>(p, B, gate, ldg, w, out, ldo, eps, st);
}
