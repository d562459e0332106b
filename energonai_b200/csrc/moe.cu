// Mixture-of-experts plumbing and the weight-streaming grouped product of generation steps.
//
//   moe_route     router logits -> chosen experts, their scores and each choice's place among its
//                 expert's rows
//   moe_plan      per-expert row counts -> a row layout in which every expert owns whole 128-row
//                 tiles (the unit of the tensor-core GEMM), the expert of every tile
//   moe_permute   token rows -> that layout
//   grouped_skinny  one product per group (an expert, or a head of an absorbed attention
//                 projection) for a handful of rows each: a pass over the weights of the groups
//                 that have rows, each weight read once
//   unit_act      the expert activation on its own (fp32 path)
//
// Gate and up projections are interleaved in blocks of 8 rows (8 gates, then their 8 ups), so
// that an epilogue holds both halves of a pair in one thread.
#include "common.cuh"
#include "gated.cuh"
#include "router.cuh"

namespace eb {
namespace {

// ---- routing of prompt-sized batches ------------------------------------------------------------
constexpr int kRouteWarps = 4;

// RULE: the choice follows `rule` (router.cuh); `experts` are the choices, those from `rule.real` on have no rows.
template <bool RULE>
__global__ void __launch_bounds__(kRouteWarps * 32)
moe_route_kernel(const float *logits, long long ld, int tokens, int experts, int top, const int *first, int rows_per_batch, int *idx,
                 float *weights, int *counts, int *ranks, const RouterRule rule, float *gate, int gate_col) {
  extern __shared__ float dyn[];
  griddep_wait();
  griddep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * kRouteWarps + warp;
  if (t >= tokens) return;
  if (first && t % rows_per_batch < first[t / rows_per_batch]) {       // a padding row: no expert
    for (int k = lane; k < top; k += 32) {
      idx[(long long)t * top + k] = -1;
      weights[(long long)t * top + k] = 0.f;
    }
    if (gate && lane == 0) gate[t] = 0.f;
    return;
  }
  float *z = dyn + warp * (RULE ? rule_floats(experts, rule) : experts);
  for (int e = lane; e < experts; e += 32) z[e] = logits[(long long)t * ld + e];
  if (gate && lane == 0) gate[t] = 1.f / (1.f + expf(-logits[(long long)t * ld + gate_col]));
  __syncwarp();
  if (RULE) route_warp_rule<false>(z, experts, top, rule, idx + (long long)t * top, weights + (long long)t * top, counts, ranks ? ranks + (long long)t * top : nullptr);
  else route_warp(z, experts, top, idx + (long long)t * top, weights + (long long)t * top, counts, ranks ? ranks + (long long)t * top : nullptr);
}

constexpr int kPlanThreads = 1024;

// counts[experts * kCountStride] -> offsets[experts] (first row of the expert, a multiple of 128), tile_group[],
// live_tiles; the counts are zeroed for the next batch.
__global__ void __launch_bounds__(kPlanThreads)
moe_plan_kernel(int *counts, int experts, int *offsets, int *tile_group, int max_tiles, int *live_tiles) {
  __shared__ int warp_tot[kPlanThreads / 32];
  griddep_wait();
  griddep_launch();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int per = (experts + kPlanThreads - 1) / kPlanThreads;
  const int e0 = tid * per, e1 = min(experts, e0 + per);
  int mine = 0;
  for (int e = e0; e < e1; ++e) mine += (counts[e * kCountStride] + 127) / 128;
  int incl = mine;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int v = __shfl_up_sync(0xffffffffu, incl, o);
    if (lane >= o) incl += v;
  }
  if (lane == 31) warp_tot[warp] = incl;
  __syncthreads();
  int before = 0, total = 0;
  for (int w = 0; w < kPlanThreads / 32; ++w) {
    if (w < warp) before += warp_tot[w];
    total += warp_tot[w];
  }
  int tile = before + incl - mine;
  for (int e = e0; e < e1; ++e) {
    const int n = (counts[e * kCountStride] + 127) / 128;
    offsets[e] = tile * 128;
    for (int i = 0; i < n; ++i)
      if (tile + i < max_tiles) tile_group[tile + i] = e;
    tile += n;
    counts[e * kCountStride] = 0;
  }
  if (tid == 0) *live_tiles = min(total, max_tiles);
}

constexpr int kPermuteThreads = 256;

// Row t of x goes to row offsets[e] + rank of every expert it chose; rows[] keeps that place.
__global__ void __launch_bounds__(kPermuteThreads)
moe_permute_kernel(const uint4 *x, long long ldx16, int packs, int tokens, int top, const int *idx, const int *ranks, const int *offsets,
                   int *rows, uint4 *out, long long ldo16, int max_rows) {
  griddep_wait();
  griddep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * (kPermuteThreads / 32) + warp;
  if (t >= tokens) return;
  const long long a0 = (long long)t * top;
  for (int k0 = 0; k0 < top; k0 += 32) {
    int dest = -1;                                 // lane k: destination of choice k0 + k
    if (k0 + lane < top) {
      const int e = idx[a0 + k0 + lane];
      const int rank = e >= 0 ? ranks[a0 + k0 + lane] : -1;
      if (rank >= 0) {                             // (a choice that stands for the input itself has no rank)
        dest = offsets[e] + rank;
        if (dest >= max_rows) dest = -1;
      }
      rows[a0 + k0 + lane] = dest;
    }
    const int n = min(32, top - k0);
    for (int c = lane; c - lane < packs; c += 32) {
      uint4 v = make_uint4(0, 0, 0, 0);
      if (c < packs) v = x[(long long)t * ldx16 + c];
      for (int k = 0; k < n; ++k) {
        const int d = __shfl_sync(0xffffffffu, dest, k);
        if (d >= 0 && c < packs) out[(long long)d * ldo16 + c] = v;
      }
    }
  }
}

// n2: columns of y (a gated unit reads twice as many, in the 8 + 8 order)
template <typename T>
__global__ void unit_act_kernel(const T *x, long long ldx, T *y, long long ldy, int n1, int n2, int unit, float limit, float alpha) {
  griddep_wait();
  griddep_launch();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)n1 * n2) return;
  const long long m = i / n2;
  const int c = (int)(i - m * n2), col = (c >> 3) * 16 + (c & 7);
  if (unit == EB_UNIT_GELU) y[m * ldy + c] = from_f32<T>(gelu_erf_value(to_f32<T>(x[m * ldx + c])));
  else y[m * ldy + c] = from_f32<T>(unit_value(unit, to_f32<T>(x[m * ldx + col]), to_f32<T>(x[m * ldx + col + 8]), limit, alpha));
}

// ---- the weight-streaming grouped product ---------------------------------------------------------
struct SkinnyParams {
  const void *A;               // row of list entry i: A + (i / a_div) * lda + group * a_gs
  long long lda, a_gs;
  int a_div;
  const void *W;               // group g: W + g * w_gs, [N][K] rows ldw apart
  long long w_gs, ldw;
  void *C;                     // row i of group g: C + i * ldc + g * c_gs
  long long ldc, c_gs;
  const int *idx;              // group of list entry i, or null: every group has all rows
  int rows;                    // list entries
  int N, K;
  int unit;
  float limit, alpha;
  int ksplit;                  // the warps of a CTA share 16 weight rows and take this many columns each (0: own rows, all columns)
};

template <typename T> __device__ __forceinline__ void mma_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1);
template <> __device__ __forceinline__ void mma_16816<__half>(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
template <> __device__ __forceinline__ void mma_16816<__nv_bfloat16>(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint4 ld_stream(const void *p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.L2::128B.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

// 16 weight rows of one warp against up to 8*NT rows of the group, K in steps of 32 per lane
// quartet: lane (g, t) loads 16 bytes of weight rows g and g + 8 and of activation row g at the
// same 8 columns, and hands them to two MMAs.  Which columns an MMA calls k = 0..15 does not
// matter as long as both operands agree, so nothing is rearranged.
// With ksplit the warps of the CTA add their parts up in shared memory, always in the same order.
template <typename T, int NT, int U, bool SPLIT>
__device__ __forceinline__ void skinny_tile(const SkinnyParams &p, int group, int row0, const int *list, int base, int n, float *part) {
  const int warp = threadIdx.x >> 5, k_begin = SPLIT ? warp * p.ksplit : 0, k_end = SPLIT ? min(p.K, k_begin + p.ksplit) : p.K;
  const int lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const T *W = reinterpret_cast<const T *>(p.W) + (long long)group * p.w_gs;
  const T *A = reinterpret_cast<const T *>(p.A) + (long long)group * p.a_gs;
  const int ra = min(row0 + g, p.N - 1), rb = min(row0 + g + 8, p.N - 1);      // rows beyond N: computed, not stored
  const T *wa = W + (long long)ra * p.ldw + t * 8, *wb = W + (long long)rb * p.ldw + t * 8;
  const T *xr[NT];
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    const int r = base + min(j * 8 + g, n - 1);
    const int i = list ? list[r] : r;
    xr[j] = A + (long long)(i / p.a_div) * p.lda + t * 8;
  }
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  for (int k0 = k_begin; k0 < k_end; k0 += 32 * U) {
    uint4 a[U], b[U], x[U][NT];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = k0 + u * 32;
      const bool ok = k + t * 8 < k_end;
      a[u] = ok ? ld_stream(wa + k) : zero;
      b[u] = ok ? ld_stream(wb + k) : zero;
#pragma unroll
      for (int j = 0; j < NT; ++j) x[u][j] = ok ? *reinterpret_cast<const uint4 *>(xr[j] + k) : zero;
    }
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        mma_16816<T>(acc[j], a[u].x, b[u].x, a[u].y, b[u].y, x[u][j].x, x[u][j].y);
        mma_16816<T>(acc[j], a[u].z, b[u].z, a[u].w, b[u].w, x[u][j].z, x[u][j].w);
      }
  }
  if (SPLIT) {
    const int warps = blockDim.x >> 5;
    __syncthreads();                               // the parts of an earlier round have been read
    if (warp > 0) {
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) part[((warp - 1) * 16 + j * 4 + e) * 32 + lane] = acc[j][e];
    }
    __syncthreads();
    if (warp > 0) return;
    for (int w = 0; w < warps - 1; ++w)
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[j][e] += part[(w * 16 + j * 4 + e) * 32 + lane];
  }
  T *C = reinterpret_cast<T *>(p.C) + (long long)group * p.c_gs;
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = j * 8 + t * 2 + e;
      if (r >= n) continue;
      const int i = list ? list[base + r] : base + r;
      T *c = C + (long long)i * p.ldc;
      if (p.unit == EB_UNIT_CLAMPED || p.unit == EB_UNIT_GEGLU) {
        if (row0 + g + 8 < p.N) c[row0 / 2 + g] = from_f32<T>(unit_value(p.unit, acc[j][e], acc[j][2 + e], p.limit, p.alpha));
      } else if (p.unit == EB_UNIT_GELU) {
        if (row0 + g < p.N) c[row0 + g] = from_f32<T>(gelu_erf_fast(acc[j][e]));
        if (row0 + g + 8 < p.N) c[row0 + g + 8] = from_f32<T>(gelu_erf_fast(acc[j][2 + e]));
      } else {
        if (row0 + g < p.N) c[row0 + g] = from_f32<T>(acc[j][e]);
        if (row0 + g + 8 < p.N) c[row0 + g + 8] = from_f32<T>(acc[j][2 + e]);
      }
    }
}

template <typename T, bool SPLIT>
__global__ void __launch_bounds__(128) grouped_skinny_kernel(const SkinnyParams p) {
  extern __shared__ int list[];
  __shared__ int s_n;
  __shared__ float part[SPLIT ? 3 * 16 * 32 : 1];
  griddep_wait();
  griddep_launch();
  const int group = blockIdx.y;
  int n = p.rows;
  if (p.idx) {
    if (threadIdx.x == 0) s_n = 0;
    __syncthreads();
    for (int i = threadIdx.x; i < p.rows; i += blockDim.x)
      if (p.idx[i] == group) list[atomicAdd(&s_n, 1)] = i;      // any order: every row is computed on its own
    __syncthreads();
    n = s_n;
  }
  const int row0 = (SPLIT ? blockIdx.x : blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5)) * 16;
  if (n == 0 || row0 >= p.N) return;
  const int *l = p.idx ? list : nullptr;
  for (int base = blockIdx.z * 32; base < n; base += 32 * gridDim.z) {
    const int m = min(32, n - base);
    if (m <= 8) skinny_tile<T, 1, 8, SPLIT>(p, group, row0, l, base, m, part);
    else if (m <= 16) skinny_tile<T, 2, 4, SPLIT>(p, group, row0, l, base, m, part);
    else skinny_tile<T, 4, 2, SPLIT>(p, group, row0, l, base, m, part);
  }
}

}  // namespace
}  // namespace eb

using namespace eb;

template <bool RULE>
static int route_impl(const float *logits, long long ld, int tokens, int experts, int top, const int32_t *first, int rows_per_batch,
                      int32_t *idx, float *weights, int32_t *counts, int32_t *ranks, const RouterRule &rule, float *gate, int gate_col, void *stream) {
  if (tokens == 0) return EB_OK;
  EB_REQUIRE(logits && idx && weights, "moe_route: null pointer");
  EB_REQUIRE(tokens > 0 && experts > 0 && experts <= kMaxExperts && top > 0 && top <= experts && ld >= experts,
             "moe_route: bad sizes (%d tokens, %d experts, top %d)", tokens, experts, top);
  EB_REQUIRE((counts == nullptr) == (ranks == nullptr), "moe_route: counts and ranks go together");
  EB_REQUIRE(!first || rows_per_batch > 0, "moe_route: first needs rows_per_batch");
  const size_t smem = (size_t)kRouteWarps * (RULE ? rule_floats(experts, rule) : experts) * sizeof(float);
  if (smem > 48 * 1024 && cudaFuncSetAttribute(moe_route_kernel<RULE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    cudaGetLastError();
    return fail(EB_ECUDA, "moe_route: cannot reserve %zu bytes of shared memory", smem);
  }
  launch_pdl(moe_route_kernel<RULE>, dim3((tokens + kRouteWarps - 1) / kRouteWarps), dim3(kRouteWarps * 32), smem, as_stream(stream), logits, ld,
             tokens, experts, top, first, rows_per_batch, idx, weights, counts, ranks, rule, gate, gate_col);
  return check_launch("moe_route");
}

extern "C" int eb_moe_route(const float *logits, long long ld, int tokens, int experts, int top, const int32_t *first, int rows_per_batch,
                            int32_t *idx, float *weights, int32_t *counts, int32_t *ranks, void *stream) {
  return route_impl<false>(logits, ld, tokens, experts, top, first, rows_per_batch, idx, weights, counts, ranks, RouterRule{}, nullptr, 0, stream);
}

extern "C" int eb_moe_route_rule(const float *logits, long long ld, int tokens, int choices, int experts, int top, const float *correction,
                                 int groups, int keep, const int32_t *first, int rows_per_batch, int32_t *idx, float *weights, int32_t *counts,
                                 int32_t *ranks, float *shared_gate, void *stream) {
  RouterRule rule;
  if (int rc = make_rule("moe_route", choices, experts, top, correction, groups, keep, &rule)) return rc;
  EB_REQUIRE(!shared_gate || ld > choices, "moe_route: the shared expert's gate is the logit behind the choices");
  return route_impl<true>(logits, ld, tokens, choices, top, first, rows_per_batch, idx, weights, counts, ranks, rule, shared_gate, choices, stream);
}

extern "C" int eb_moe_plan(int32_t *counts, int experts, int32_t *offsets, int32_t *tile_group, int max_tiles, int32_t *live_tiles,
                           void *stream) {
  EB_REQUIRE(counts && offsets && tile_group && live_tiles, "moe_plan: null pointer");
  EB_REQUIRE(experts > 0 && experts <= kMaxExperts && max_tiles > 0, "moe_plan: bad sizes");
  launch_pdl(moe_plan_kernel, dim3(1), dim3(kPlanThreads), 0, as_stream(stream), counts, experts, offsets, tile_group, max_tiles, live_tiles);
  return check_launch("moe_plan");
}

extern "C" int eb_moe_permute(const void *x, long long ldx, int n2, int dtype, int tokens, int top, const int32_t *idx,
                              const int32_t *ranks, const int32_t *offsets, int32_t *rows, void *out, long long ldo, int max_rows,
                              void *stream) {
  if (tokens == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "moe_permute: bad dtype %d", dtype);
  EB_REQUIRE(x && idx && ranks && offsets && rows && out, "moe_permute: null pointer");
  const int per = 16 / dtype_size(dtype);
  EB_REQUIRE(n2 > 0 && n2 % per == 0 && ldx % per == 0 && ldo % per == 0 && ldx >= n2 && ldo >= n2, "moe_permute: rows must be whole 16-byte packs");
  EB_REQUIRE(aligned16(x) && aligned16(out), "moe_permute: pointers must be 16-byte aligned");
  EB_REQUIRE(tokens > 0 && top > 0 && max_rows > 0, "moe_permute: bad sizes");
  launch_pdl(moe_permute_kernel, dim3((tokens + 7) / 8), dim3(kPermuteThreads), 0, as_stream(stream), reinterpret_cast<const uint4 *>(x),
             ldx / per, n2 / per, tokens, top, idx, ranks, offsets, rows, reinterpret_cast<uint4 *>(out), ldo / per, max_rows);
  return check_launch("moe_permute");
}

extern "C" int eb_unit_act(const void *x, long long ldx, void *y, long long ldy, int n1, int n2, int unit, float limit, float alpha, int dtype,
                           void *stream) {
  if (n1 == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype) && x && y, "unit_act: bad dtype or null pointer");
  EB_REQUIRE(unit >= EB_UNIT_CLAMPED && unit <= EB_UNIT_GELU, "unit_act: unknown unit %d", unit);
  EB_REQUIRE(n1 > 0 && n2 > 0 && n2 % 8 == 0 && ldx >= (unit == EB_UNIT_GELU ? n2 : 2 * n2) && ldy >= n2, "unit_act: bad sizes");
  const long long total = (long long)n1 * n2;
  EB_REQUIRE((total + 255) / 256 < (1ll << 31), "unit_act: too many elements");
  const dim3 g((unsigned)((total + 255) / 256)), b(256);
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F32) launch_pdl(unit_act_kernel<float>, g, b, 0, st, (const float *)x, ldx, (float *)y, ldy, n1, n2, unit, limit, alpha);
  else if (dtype == EB_F16) launch_pdl(unit_act_kernel<__half>, g, b, 0, st, (const __half *)x, ldx, (__half *)y, ldy, n1, n2, unit, limit, alpha);
  else launch_pdl(unit_act_kernel<__nv_bfloat16>, g, b, 0, st, (const __nv_bfloat16 *)x, ldx, (__nv_bfloat16 *)y, ldy, n1, n2, unit, limit, alpha);
  return check_launch("unit_act");
}

extern "C" int eb_gated_act(const void *x, long long ldx, void *y, long long ldy, int n1, int half, float limit, float alpha, int dtype,
                            void *stream) {
  return eb_unit_act(x, ldx, y, ldy, n1, half, EB_UNIT_CLAMPED, limit, alpha, dtype, stream);
}

extern "C" int eb_grouped_skinny(const void *A, long long lda, long long a_group_stride, int a_div, const void *W, long long w_group_stride,
                                 long long ldw, void *C, long long ldc, long long c_group_stride, const int32_t *idx, int rows, int groups,
                                 int N, int K, int unit, float limit, float alpha, int dtype, void *stream) {
  if (rows == 0 || groups == 0) return EB_OK;
  const bool gated = unit == EB_UNIT_CLAMPED || unit == EB_UNIT_GEGLU;
  EB_REQUIRE(unit >= EB_UNIT_NONE && unit <= EB_UNIT_GELU, "grouped_skinny: unknown unit %d", unit);
  EB_REQUIRE(dtype == EB_F16 || dtype == EB_BF16, "grouped_skinny: fp16 or bf16 only (dtype %d)", dtype);
  EB_REQUIRE(A && W && C, "grouped_skinny: null pointer");
  EB_REQUIRE(rows > 0 && groups > 0 && groups <= 65535 && N > 0 && K > 0 && a_div > 0, "grouped_skinny: bad sizes");
  EB_REQUIRE(K % 8 == 0 && lda % 8 == 0 && ldw % 8 == 0 && a_group_stride % 8 == 0 && w_group_stride % 8 == 0 && ldw >= K && lda >= 0,
             "grouped_skinny: K and the strides of A and W must be multiples of 8");
  EB_REQUIRE(!gated || N % 16 == 0, "grouped_skinny: a gated product needs N a multiple of 16");
  EB_REQUIRE(aligned16(A) && aligned16(W), "grouped_skinny: pointers must be 16-byte aligned");
  EB_REQUIRE(!idx || rows <= 10240, "grouped_skinny: at most 10240 list entries (got %d)", rows);
  SkinnyParams p{};
  p.A = A; p.lda = lda; p.a_gs = a_group_stride; p.a_div = a_div; p.W = W; p.w_gs = w_group_stride; p.ldw = ldw;
  p.C = C; p.ldc = ldc; p.c_gs = c_group_stride; p.idx = idx; p.rows = rows; p.N = N; p.K = K;
  p.unit = unit; p.limit = limit; p.alpha = alpha;
  // Too few strips to give every SM a CTA of four: with many columns the four warps share a strip
  // and split its columns, with few the CTAs get fewer warps.  (The choice depends on the weights'
  // shape alone, so a row's result does not change with the batch.)
  const int strips = (N + 15) / 16;
  int warps = 4;
  const bool few = (long long)((strips + warps - 1) / warps) * groups < 2ll * sm_count(), split = few && K >= 256;
  if (split) p.ksplit = ((K + warps - 1) / warps + 31) / 32 * 32;
  while (!split && warps > 1 && (long long)((strips + warps - 1) / warps) * groups < 2ll * sm_count()) warps >>= 1;
  // (groups without a list: the rows come 32 to a CTA, side by side)
  const dim3 g(split ? strips : (strips + warps - 1) / warps, groups, idx ? 1 : (rows + 31) / 32), b(warps * 32);
  const size_t smem = idx ? (size_t)rows * sizeof(int) : 0;
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F16) launch_pdl(split ? grouped_skinny_kernel<__half, true> : grouped_skinny_kernel<__half, false>, g, b, smem, st, p);
  else launch_pdl(split ? grouped_skinny_kernel<__nv_bfloat16, true> : grouped_skinny_kernel<__nv_bfloat16, false>, g, b, smem, st, p);
  return check_launch("grouped_skinny");
}
