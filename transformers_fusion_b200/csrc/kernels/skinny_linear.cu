// Products of few rows (decode steps): out[M, N] = act(x[M, K] . W[N, K]^T [+ bias]) for M <= 64 in bf16 with fp32 accumulation, one launch
// and no workspace.  A 128-row tcgen05 tile would be mostly padding and its split-K form needs a second kernel; here a block
// takes 16 columns, its eight warps share the reduction dimension, and the weights go from global memory to the operand registers of
// mma.sync without a stop: both operands may be read in the same permuted order of k, so a lane takes 16 consecutive entries of a
// row (32 bytes) and calls them the k slots that it owns in four consecutive steps.
// The same kernel runs one such product per head (grid y) over slices of x, with an optional gate per row and head.
#include "tfb_elem.cuh"
#include "tfb_host.h"
#include "tfb_mma.cuh"

namespace tfb {

constexpr int SK_N = 16, SK_WARPS = 8;

struct SkinnyArgs {
  const __nv_bfloat16 *x, *w;
  long long ldx, ldw;
  void* out;
  long long ldo;
  int M, N, K, act, out_f32;
  int x_head, out_head;             // entries between the heads of x and of out; W advances by N rows
  const __nv_bfloat16* gate;        // [M, ldg] or null: head h is multiplied by sigmoid(gate[:, h])
  long long ldg;
  const __nv_bfloat16* bias;        // [N] or null
};

struct Row16 { uint32_t u[8]; };      // 16 consecutive entries of a row
__device__ __forceinline__ Row16 load16(const __nv_bfloat16* row, int k, int K, bool live) {      // K is a multiple of 8
  Row16 r;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  const uint4 a = live && k < K ? *reinterpret_cast<const uint4*>(row + k) : zero;
  const uint4 b = live && k + 8 < K ? *reinterpret_cast<const uint4*>(row + k + 8) : zero;
  r.u[0] = a.x; r.u[1] = a.y; r.u[2] = a.z; r.u[3] = a.w;
  r.u[4] = b.x; r.u[5] = b.y; r.u[6] = b.z; r.u[7] = b.w;
  return r;
}

template <int MT>
__global__ void __launch_bounds__(SK_WARPS * 32) skinny_linear_kernel(const SkinnyArgs p) {
  tfb::pdl_sync();
  __shared__ float red[SK_WARPS][MT * 16][SK_N + 1];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, q = lane & 3;
  const int n0 = blockIdx.x * SK_N, h = blockIdx.y, m0 = blockIdx.z * MT * 16, M = min(MT * 16, p.M - m0);
  float acc[MT][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 2; ++n) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.f;
  const __nv_bfloat16* w0 = p.w + ((long long)h * p.N + n0 + g) * p.ldw;
  const __nv_bfloat16* x0 = p.x + (m0 + g) * p.ldx + (long long)h * p.x_head;
#pragma unroll 2
  for (int k0 = warp * 64; k0 < p.K; k0 += SK_WARPS * 64) {
    const int k = k0 + q * 16;
    Row16 b[2];
#pragma unroll
    for (int n = 0; n < 2; ++n) b[n] = load16(w0 + n * 8 * p.ldw, k, p.K, n0 + n * 8 + g < p.N);
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const Row16 a0 = load16(x0 + m * 16 * p.ldx, k, p.K, m * 16 + g < M), a1 = load16(x0 + (m * 16 + 8) * p.ldx, k, p.K, m * 16 + 8 + g < M);
#pragma unroll
      for (int s = 0; s < 4; ++s) {
        const uint32_t a[4] = {a0.u[2 * s], a1.u[2 * s], a0.u[2 * s + 1], a1.u[2 * s + 1]};
#pragma unroll
        for (int n = 0; n < 2; ++n) mma_bf16(acc[m][n], a, b[n].u[2 * s], b[n].u[2 * s + 1]);
      }
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) red[warp][m * 16 + g + (e >> 1) * 8][n * 8 + q * 2 + (e & 1)] = acc[m][n][e];
  __syncthreads();
  for (int i = threadIdx.x; i < MT * 16 * SK_N; i += SK_WARPS * 32) {
    const int m = i / SK_N, n = i % SK_N;
    if (m >= M || n0 + n >= p.N) continue;
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < SK_WARPS; ++w) v += red[w][m][n];
    if (p.bias) v += __bfloat162float(p.bias[n0 + n]);
    if (p.act == 4) {
      v = fmaxf(v, 0.f);
      v *= v;
    }
    if (p.gate) v *= 1.f / (1.f + expf(-__bfloat162float(p.gate[(m0 + m) * p.ldg + h])));
    const long long at = (m0 + m) * p.ldo + (long long)h * p.out_head + n0 + n;
    if (p.out_f32) static_cast<float*>(p.out)[at] = v;
    else static_cast<__nv_bfloat16*>(p.out)[at] = __float2bfloat16(v);
  }
}

}  // namespace tfb

using bf16 = __nv_bfloat16;

// 16-row, 16-column blocks x their depth: every block reads its rows and columns of both operands
static long long tfb_skinny_work(int M, long long N, int K) { return (N + 15) / 16 * ((M + 15) / 16) * K; }

static int launch_skinny(const tfb::SkinnyArgs& p, int heads, int rows, void* stream) {
  using namespace tfb;
  if (p.M <= 0 || p.N <= 0 || p.K <= 0 || p.K % 8 || p.ldx % 8 || p.ldw % 8 || p.x_head % 8 || heads <= 0 || heads > 65535 || p.M > 16 * 65535 ||
      (reinterpret_cast<uintptr_t>(p.x) & 15) || (reinterpret_cast<uintptr_t>(p.w) & 15))
    return TFB_ERR_ARG;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (rows == 0) rows = p.M <= 16 || tfb_skinny_work(p.M, p.N * heads, p.K) <= 1500000 ? 16 : 32;
  const dim3 grid((p.N + SK_N - 1) / SK_N, heads, (p.M + rows - 1) / rows);
  if (rows == 16) launch_k(skinny_linear_kernel<1>, grid, SK_WARPS * 32, 0, st, p);
  else if (rows == 32) launch_k(skinny_linear_kernel<2>, grid, SK_WARPS * 32, 0, st, p);
  else if (rows == 64) launch_k(skinny_linear_kernel<4>, grid, SK_WARPS * 32, 0, st, p);
  else return TFB_ERR_ARG;
  return int(cudaGetLastError());
}

// 1 where the few-row form is the one to take.  Measured against the tcgen05 form (with its split-K finalize): it wins while a warp's share
// of K is short and, for more than 16 rows, while reading the operands once per block stays cheap.
TFB_API int tfb_skinny_fits(int M, int N, int K) {
  return M <= 64 && K % 8 == 0 && K <= 6144 && (M <= 16 || tfb_skinny_work(M, N, K) <= 2000000);
}

// act: 0 none, 4 relu squared.  rows: rows of a block (16, 32 or 64; 0: the kernel's choice).  Row pitches are multiples of 8 entries, x and w aligned to 16 bytes.
TFB_API int tfb_skinny_linear(const void* x, long long ldx, const void* w, long long ldw, void* out, long long ldo, int M, int N, int K, int act,
                              int out_f32, int rows, const void* bias, void* stream) {
  if (M > 64 || (act != 0 && act != 4)) return TFB_ERR_ARG;
  return launch_skinny(tfb::SkinnyArgs{static_cast<const bf16*>(x), static_cast<const bf16*>(w), ldx, ldw, out, ldo, M, N, K, act, out_f32, 0, 0,
                                       nullptr, 0, static_cast<const bf16*>(bias)}, 1, rows, stream);
}

// One product per head: x [M, ldx] (x_head entries between heads), w: heads blocks [N, K] stacked on the rows, out [M, ldo] (N entries per
// head), gate [M, ldg] or null.
TFB_API int tfb_skinny_linear_heads(const void* x, long long ldx, int x_head, const void* w, long long ldw, void* out, long long ldo, const void* gate,
                                    long long ldg, int M, int heads, int N, int K, int rows, void* stream) {
  return launch_skinny(tfb::SkinnyArgs{static_cast<const bf16*>(x), static_cast<const bf16*>(w), ldx, ldw, out, ldo, M, N, K, 0, 0, x_head, N,
                                       static_cast<const bf16*>(gate), ldg, nullptr}, heads, rows, stream);
}
