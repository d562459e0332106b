// C = A . W^T with fp32 operands and plain fp32 multiply-adds (no reduced-precision tensor mode):
// the product of models that are run in true 32-bit.  A tiled CUDA-core kernel, 64 x 64 outputs per
// CTA.  Groups, two ways:
//   tile_group != null   the rows of A come in 128-row tiles, tile i using the weights of group
//                        tile_group[i]; tiles from *live_tiles on are skipped
//   groups > 1           blockIdx.z = group: strides between the groups' operands
// A single product may add a bias and apply xIELU to its first columns.
#include "common.cuh"
#include "xielu.cuh"

namespace eb {
namespace {

constexpr int kT = 64, kStep = 16, kF32Threads = 256;

struct F32Params {
  const float *A, *W;
  float *C;
  long long lda, ldw, ldc, a_gs, w_gs, c_gs;
  int M, N, K;
  const int *tile_group, *live_tiles;
  const float *bias, *act_params;   // both or either may be null; xIELU on the columns below act_cols
  int act_cols;
};

__global__ void __launch_bounds__(kF32Threads) gemm_f32_kernel(const F32Params p) {
  __shared__ float sa[kStep][kT + 4], sw[kStep][kT + 4];
  griddep_wait();
  griddep_launch();
  const int m0 = blockIdx.y * kT, n0 = blockIdx.x * kT;
  long long group = blockIdx.z;
  if (p.tile_group) {
    const int tile = m0 / 128;
    if (tile >= *p.live_tiles) return;
    group = p.tile_group[tile];
  }
  const float *A = p.A + (p.tile_group ? 0 : group * p.a_gs), *W = p.W + group * p.w_gs;
  float *C = p.C + (p.tile_group ? 0 : group * p.c_gs);
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += kStep) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = threadIdx.x + i * kF32Threads, r = e / kStep, k = e % kStep;
      sa[k][r] = (m0 + r < p.M && k0 + k < p.K) ? A[(long long)(m0 + r) * p.lda + k0 + k] : 0.f;
      sw[k][r] = (n0 + r < p.N && k0 + k < p.K) ? W[(long long)(n0 + r) * p.ldw + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kStep; ++k) {
      float a[4], w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = sa[k][ty * 4 + i]; w[i] = sw[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
    }
    __syncthreads();
  }
  float up = 0.f, down = 0.f;
  if (p.act_params) { up = p.act_params[0]; down = p.act_params[1]; }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m >= p.M || n >= p.N) continue;
      float v = acc[i][j] + (p.bias ? p.bias[n] : 0.f);
      if (p.act_params && n < p.act_cols) v = xielu_exact(v, up, down);
      C[(long long)m * p.ldc + n] = v;
    }
}

}  // namespace
}  // namespace eb

using namespace eb;

extern "C" int eb_gemm_f32(const float *A, long long lda, long long a_group_stride, const float *W, long long ldw, long long w_group_stride,
                           float *C, long long ldc, long long c_group_stride, int M, int N, int K, int groups, const int32_t *tile_group,
                           const int32_t *live_tiles, const float *bias, int act_cols, const float *act_params, void *stream) {
  if (M == 0 || N == 0 || groups == 0) return EB_OK;
  EB_REQUIRE(A && W && C, "gemm_f32: null pointer");
  EB_REQUIRE(M > 0 && N > 0 && K > 0 && groups > 0 && groups <= 65535, "gemm_f32: bad sizes");
  EB_REQUIRE(lda >= K && ldw >= K && ldc >= N, "gemm_f32: leading dimensions smaller than the rows they hold");
  EB_REQUIRE((tile_group == nullptr) == (live_tiles == nullptr) && (!tile_group || groups == 1),
             "gemm_f32: tile_group goes with live_tiles and without strided groups");
  EB_REQUIRE((!bias && !act_params) || (groups == 1 && !tile_group), "gemm_f32: bias and activation belong to a single product");
  EB_REQUIRE((M + kT - 1) / kT <= 65535, "gemm_f32: too many rows");
  F32Params p{};
  p.A = A; p.W = W; p.C = C; p.lda = lda; p.ldw = ldw; p.ldc = ldc; p.a_gs = a_group_stride; p.w_gs = w_group_stride; p.c_gs = c_group_stride;
  p.M = M; p.N = N; p.K = K; p.tile_group = tile_group; p.live_tiles = live_tiles;
  p.bias = bias; p.act_cols = act_cols; p.act_params = act_params;
  launch_pdl(gemm_f32_kernel, dim3((N + kT - 1) / kT, (M + kT - 1) / kT, groups), dim3(kF32Threads), 0, as_stream(stream), p);
  return check_launch("gemm_f32");
}
