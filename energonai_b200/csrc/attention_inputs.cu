// What lies between the projection of an attention layer and the attention itself, one row per CTA:
// RMS norm of the whole query and of the whole key (before they are heads), a query temperature that
// grows with the position, values mixed with those an earlier layer cached for the same token, and the
// stores into the key / value cache.  Statistics and factors are fp32.
#include "common.cuh"

namespace eb {
namespace {

struct InputParams {
  const void *proj;
  long long ldp;
  int nq, nk, nv;              // columns of q, k, v
  const void *wq, *wk;
  float inv_q, inv_k, eps, coef;
  int every;
  const float *vmix;
  const void *vf;
  long long vf_bs, vf_rs;
  void *q;
  long long ldq;
  void *k, *v;
  long long k_bs, k_rs, v_bs, v_rs;
  int cache_rows, rows_per_batch;
  const int *pos_dev, *first;
};

template <typename T> struct Pack8 {               // 8 elements of T
  static constexpr int N = Vec16<T>::N;
  Vec16<T> part[8 / N];
  __device__ __forceinline__ void load(const T *p) {
#pragma unroll
    for (int i = 0; i < 8 / N; ++i) part[i].load(p + i * N);
  }
  __device__ __forceinline__ void unpack(float (&f)[8]) const {
#pragma unroll
    for (int i = 0; i < 8 / N; ++i) {
      float t[N];
      part[i].unpack(t);
#pragma unroll
      for (int e = 0; e < N; ++e) f[i * N + e] = t[e];
    }
  }
  static __device__ __forceinline__ void store(T *p, const float (&f)[8]) {
#pragma unroll
    for (int i = 0; i < 8 / N; ++i) {
      Vec16<T> a;
      float t[N];
#pragma unroll
      for (int e = 0; e < N; ++e) t[e] = f[i * N + e];
      a.pack(t);
      a.store(p + i * N);
    }
  }
};

// PACKS packs of 8 columns per thread stay in registers, beside what each is multiplied by or mixed
// with: everything a row needs is requested before the two sums are formed.
template <typename T, int PACKS, int THREADS>
__global__ void __launch_bounds__(THREADS) attention_inputs_kernel(const InputParams p) {
  __shared__ float2 scratch[THREADS / 32];
  griddep_wait();
  griddep_launch();
  const long long row = blockIdx.x;
  const long long b = row / p.rows_per_batch;
  const int col = (p.pos_dev ? *p.pos_dev : 0) + (int)(row - b * p.rows_per_batch);
  const T *x = reinterpret_cast<const T *>(p.proj) + row * p.ldp;
  const int nq = p.nq / 8, nk = p.nk / 8, all = nq + nk + p.nv / 8;
  const bool keep = col >= 0 && col < p.cache_rows;
  const T *vf = p.vmix && keep ? reinterpret_cast<const T *>(p.vf) + b * p.vf_bs + (long long)col * p.vf_rs : nullptr;
  Pack8<T> xv[PACKS], wv[PACKS];
#pragma unroll
  for (int i = 0; i < PACKS; ++i) {
    const int c = threadIdx.x + i * THREADS;
    if (c >= all) break;
    xv[i].load(x + c * 8);
    if (c < nq) wv[i].load(reinterpret_cast<const T *>(p.wq) + c * 8);
    else if (c < nq + nk) wv[i].load(reinterpret_cast<const T *>(p.wk) + (c - nq) * 8);
    else if (vf) wv[i].load(vf + (c - nq - nk) * 8);
  }
  const float lambda = vf ? *p.vmix : 0.f;
  const int first = p.first ? p.first[b] : 0;
  float2 sq = make_float2(0.f, 0.f);
#pragma unroll
  for (int i = 0; i < PACKS; ++i) {
    const int c = threadIdx.x + i * THREADS;
    if (c >= nq + nk) break;
    float f[8], s = 0.f;
    xv[i].unpack(f);
#pragma unroll
    for (int e = 0; e < 8; ++e) s = fmaf(f[e], f[e], s);
    if (c < nq) sq.x += s; else sq.y += s;
  }
  sq.x = warp_sum(sq.x);
  sq.y = warp_sum(sq.y);
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = sq;
  __syncthreads();
  sq = make_float2(0.f, 0.f);
#pragma unroll
  for (int i = 0; i < THREADS / 32; ++i) {
    sq.x += scratch[i].x;
    sq.y += scratch[i].y;
  }
  float rq = rsqrtf(sq.x * p.inv_q + p.eps);
  const float rk = rsqrtf(sq.y * p.inv_k + p.eps);
  if (p.every > 0) rq *= 1.f + p.coef * logf((float)((max(0, col - first) + 1) / p.every + 1));
  T *q = reinterpret_cast<T *>(p.q) + row * p.ldq;
  T *k = reinterpret_cast<T *>(p.k) + b * p.k_bs + (long long)col * p.k_rs;
  T *v = reinterpret_cast<T *>(p.v) + b * p.v_bs + (long long)col * p.v_rs;
#pragma unroll
  for (int i = 0; i < PACKS; ++i) {
    const int c = threadIdx.x + i * THREADS;
    if (c >= all) break;
    float f[8], w[8];
    xv[i].unpack(f);
    wv[i].unpack(w);
    if (c < nq) {
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] *= rq * w[e];
      Pack8<T>::store(q + c * 8, f);
    } else if (c < nq + nk) {
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] *= rk * w[e];
      if (keep) Pack8<T>::store(k + (c - nq) * 8, f);
    } else {
      if (vf) {
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = fmaf(lambda, w[e], (1.f - lambda) * f[e]);
      }
      if (keep) Pack8<T>::store(v + (c - nq - nk) * 8, f);
    }
  }
}

template <typename T> int launch_inputs(const InputParams &p, int n1, cudaStream_t st) {
  const int packs = (p.nq + p.nk + p.nv) / 8;
  const dim3 g(n1);
  if (packs <= 128) launch_pdl(attention_inputs_kernel<T, 1, 128>, g, dim3(128), 0, st, p);
  else if (packs <= 256) launch_pdl(attention_inputs_kernel<T, 1, 256>, g, dim3(256), 0, st, p);
  else if (packs <= 512) launch_pdl(attention_inputs_kernel<T, 2, 256>, g, dim3(256), 0, st, p);
  else if (packs <= 1024) launch_pdl(attention_inputs_kernel<T, 4, 256>, g, dim3(256), 0, st, p);
  else if (packs <= 2048) launch_pdl(attention_inputs_kernel<T, 4, 512>, g, dim3(512), 0, st, p);
  else if (packs <= 4096) launch_pdl(attention_inputs_kernel<T, 4, 1024>, g, dim3(1024), 0, st, p);
  else return fail(EB_EUNSUPPORTED, "attention_inputs: %d columns are too many (32768)", packs * 8);
  return check_launch("attention_inputs");
}

// ---- keys and values for a cache with kept first positions ----
struct ValueParams {
  const void *k;
  void *v;                     // column ranges of rows ld apart; v is normalised in place
  long long ld;
  int heads, dk, dv;
  float inv_count, eps;
  void *kc, *vc;               // cache row 0: `keep` rows of the first positions, then the ring
  long long k_bs, k_rs, v_bs, v_rs;
  int keep, ring_rows, n1, rows_per_batch;
  const int *pos_dev, *first;
};

// A warp per (row, key / value head): the value over its root mean square, then key and value to the cache.
template <typename T>
__global__ void __launch_bounds__(256) attention_values_kernel(const ValueParams p) {
  griddep_wait();
  griddep_launch();
  constexpr int N = Vec16<T>::N;
  const int lane = threadIdx.x & 31;
  const long long unit = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), row = unit / p.heads;
  if (row >= p.n1) return;
  const int h = (int)(unit - row * p.heads);
  const long long b = row / p.rows_per_batch;
  const int s = (int)(row - b * p.rows_per_batch), col = (p.pos_dev ? *p.pos_dev : 0) + s, at = col - (p.first ? p.first[b] : 0);
  const bool in_ring = col >= 0 && p.rows_per_batch - s <= p.ring_rows, kept = at >= 0 && at < p.keep;
  const long long ring = p.keep + (in_ring ? col % p.ring_rows : 0);
  T *v = reinterpret_cast<T *>(p.v) + row * p.ld + h * p.dv;
  T *kc = reinterpret_cast<T *>(p.kc) + b * p.k_bs + h * p.dk, *vc = reinterpret_cast<T *>(p.vc) + b * p.v_bs + h * p.dv;
  float sq = 0.f;
  for (int i = lane * N; i < p.dv; i += 32 * N) {
    Vec16<T> w;
    float f[N];
    w.load(v + i);
    w.unpack(f);
#pragma unroll
    for (int e = 0; e < N; ++e) sq = fmaf(f[e], f[e], sq);
  }
  const float r = 1.f / sqrtf(warp_sum(sq) * p.inv_count + p.eps);
  for (int i = lane * N; i < p.dv; i += 32 * N) {
    Vec16<T> w;
    float f[N];
    w.load(v + i);
    w.unpack(f);
#pragma unroll
    for (int e = 0; e < N; ++e) f[e] *= r;
    w.pack(f);
    w.store(v + i);
    if (in_ring) w.store(vc + ring * p.v_rs + i);
    if (kept) w.store(vc + at * p.v_rs + i);
  }
  if (!in_ring && !kept) return;
  const T *k = reinterpret_cast<const T *>(p.k) + row * p.ld + h * p.dk;
  for (int i = lane * N; i < p.dk; i += 32 * N) {
    Vec16<T> w;
    w.load(k + i);
    if (in_ring) w.store(kc + ring * p.k_rs + i);
    if (kept) w.store(kc + at * p.k_rs + i);
  }
}

// ---- a gate on the concatenated heads ----
template <typename T>
__global__ void __launch_bounds__(256) sigmoid_gate_kernel(const T *y, long long ldy, const T *g, long long ldg, T *out, long long ldo, int n1, int n2) {
  griddep_wait();
  griddep_launch();
  constexpr int N = Vec16<T>::N;
  const long long per = n2 / N;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n1 * per; i += (long long)gridDim.x * blockDim.x) {
    const long long row = i / per, c = (i - row * per) * N;
    Vec16<T> a, b;
    float fa[N], fb[N];
    a.load(y + row * ldy + c);
    b.load(g + row * ldg + c);
    a.unpack(fa);
    b.unpack(fb);
#pragma unroll
    for (int e = 0; e < N; ++e) fa[e] /= 1.f + expf(-fb[e]);
    a.pack(fa);
    a.store(out + row * ldo + c);
  }
}

}  // namespace
}  // namespace eb

using namespace eb;

extern "C" int eb_attention_inputs(const void *proj, long long ldp, int heads, int kv_heads, int dk, int dv, const void *q_norm, int q_count,
                                   const void *k_norm, int k_count, float eps, float temp_coef, int temp_every, const float *vmix,
                                   const void *v_first, long long vf_batch_stride, long long vf_row_stride, void *q_out, long long ldq,
                                   void *k_cache, long long k_batch_stride, long long k_row_stride, void *v_cache, long long v_batch_stride,
                                   long long v_row_stride, int cache_rows, int n1, int rows_per_batch, const int32_t *pos_device,
                                   const int32_t *first, int dtype, void *stream) {
  if (n1 == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "attention_inputs: bad dtype %d", dtype);
  EB_REQUIRE(proj && q_norm && k_norm && q_out && k_cache && v_cache, "attention_inputs: null pointer");
  EB_REQUIRE(heads > 0 && kv_heads > 0 && dk > 0 && dv > 0 && dk % 8 == 0 && dv % 8 == 0, "attention_inputs: head sizes must be multiples of 8 (%d, %d)", dk, dv);
  EB_REQUIRE((long long)heads * dk < (1 << 24) && (long long)kv_heads * (dk > dv ? dk : dv) < (1 << 24), "attention_inputs: too many columns");
  const int nq = heads * dk, nk = kv_heads * dk, nv = kv_heads * dv;
  EB_REQUIRE(q_count > 0 && q_count <= nq && k_count > 0 && k_count <= nk, "attention_inputs: the means are over 1..all columns");
  EB_REQUIRE(temp_every >= 0 && (!vmix || v_first), "attention_inputs: bad temperature step, or a mix without the other values");
  EB_REQUIRE(n1 > 0 && rows_per_batch > 0 && n1 % rows_per_batch == 0 && cache_rows > 0, "attention_inputs: bad row counts");
  const long long strides[] = {ldp, ldq, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride, vmix ? vf_batch_stride : 0, vmix ? vf_row_stride : 0};
  for (long long s : strides) EB_REQUIRE(s % 8 == 0, "attention_inputs: strides must be multiples of 8 elements");
  EB_REQUIRE(ldp >= nq + nk + nv && ldq >= nq && k_row_stride >= nk && v_row_stride >= nv, "attention_inputs: row strides smaller than the rows they hold");
  EB_REQUIRE(aligned16(proj) && aligned16(q_norm) && aligned16(k_norm) && aligned16(q_out) && aligned16(k_cache) && aligned16(v_cache) &&
                 aligned16(v_first), "attention_inputs: pointers must be 16-byte aligned");
  InputParams p{};
  p.proj = proj; p.ldp = ldp; p.nq = nq; p.nk = nk; p.nv = nv; p.wq = q_norm; p.wk = k_norm;
  p.inv_q = 1.f / (float)q_count; p.inv_k = 1.f / (float)k_count; p.eps = eps; p.coef = temp_coef; p.every = temp_every;
  p.vmix = vmix; p.vf = v_first; p.vf_bs = vf_batch_stride; p.vf_rs = vf_row_stride;
  p.q = q_out; p.ldq = ldq; p.k = k_cache; p.k_bs = k_batch_stride; p.k_rs = k_row_stride; p.v = v_cache; p.v_bs = v_batch_stride; p.v_rs = v_row_stride;
  p.cache_rows = cache_rows; p.rows_per_batch = rows_per_batch; p.pos_dev = pos_device; p.first = first;
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F32) return launch_inputs<float>(p, n1, st);
  if (dtype == EB_F16) return launch_inputs<__half>(p, n1, st);
  return launch_inputs<__nv_bfloat16>(p, n1, st);
}

extern "C" int eb_attention_values(const void *k, void *v, long long ld, int kv_heads, int dk, int dv, int dv_count, float eps, void *k_cache,
                                   long long k_batch_stride, long long k_row_stride, void *v_cache, long long v_batch_stride, long long v_row_stride,
                                   int keep, int ring_rows, int n1, int rows_per_batch, const int32_t *pos_device, const int32_t *first, int dtype,
                                   void *stream) {
  if (n1 == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "attention_values: bad dtype %d", dtype);
  EB_REQUIRE(k && v && k_cache && v_cache, "attention_values: null pointer");
  EB_REQUIRE(kv_heads > 0 && dk > 0 && dk % 8 == 0 && dv > 0 && dv % 8 == 0 && dv_count > 0 && dv_count <= dv, "attention_values: head sizes must be multiples of 8 (%d, %d)", dk, dv);
  EB_REQUIRE(n1 > 0 && rows_per_batch > 0 && n1 % rows_per_batch == 0 && keep >= 0 && ring_rows > 0, "attention_values: bad row counts");
  const long long strides[] = {ld, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride};
  for (long long s : strides) EB_REQUIRE(s % 8 == 0, "attention_values: strides must be multiples of 8 elements");
  EB_REQUIRE(ld >= (long long)kv_heads * dk && ld >= (long long)kv_heads * dv && k_row_stride >= (long long)kv_heads * dk && v_row_stride >= (long long)kv_heads * dv,
             "attention_values: row strides smaller than the rows they hold");
  EB_REQUIRE(aligned16(k) && aligned16(v) && aligned16(k_cache) && aligned16(v_cache), "attention_values: pointers must be 16-byte aligned");
  ValueParams p{};
  p.k = k; p.v = v; p.ld = ld; p.heads = kv_heads; p.dk = dk; p.dv = dv; p.inv_count = 1.f / (float)dv_count; p.eps = eps; p.kc = k_cache; p.vc = v_cache;
  p.k_bs = k_batch_stride; p.k_rs = k_row_stride; p.v_bs = v_batch_stride; p.v_rs = v_row_stride; p.keep = keep; p.ring_rows = ring_rows; p.n1 = n1;
  p.rows_per_batch = rows_per_batch; p.pos_dev = pos_device; p.first = first;
  cudaStream_t st = as_stream(stream);
  const long long warps = (long long)n1 * kv_heads, per = warps < 8ll * sm_count() ? 1 : 8;       // few rows: a warp per CTA
  const dim3 g((unsigned)((warps + per - 1) / per)), t((unsigned)(32 * per));
  if (dtype == EB_F32) launch_pdl(attention_values_kernel<float>, g, t, 0, st, p);
  else if (dtype == EB_F16) launch_pdl(attention_values_kernel<__half>, g, t, 0, st, p);
  else launch_pdl(attention_values_kernel<__nv_bfloat16>, g, t, 0, st, p);
  return check_launch("attention_values");
}

extern "C" int eb_sigmoid_gate(const void *y, long long ldy, const void *g, long long ldg, void *out, long long ldo, int n1, int n2, int dtype,
                               void *stream) {
  if (n1 == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "sigmoid_gate: bad dtype %d", dtype);
  EB_REQUIRE(y && g && out && aligned16(y) && aligned16(g) && aligned16(out), "sigmoid_gate: null or misaligned pointer");
  EB_REQUIRE(n1 > 0 && n2 > 0 && n2 % 8 == 0 && ldy >= n2 && ldg >= n2 && ldo >= n2 && ldy % 8 == 0 && ldg % 8 == 0 && ldo % 8 == 0,
             "sigmoid_gate: rows of a multiple of 8 columns");
  cudaStream_t st = as_stream(stream);
  const long long packs = (long long)n1 * n2 / (dtype == EB_F32 ? 4 : 8), blocks = (packs + 255) / 256;
  const dim3 grid((unsigned)(blocks < 16ll * sm_count() ? blocks : 16ll * sm_count())), t(256);
#define EB_GATE(T) launch_pdl(sigmoid_gate_kernel<T>, grid, t, 0, st, (const T *)y, ldy, (const T *)g, ldg, (T *)out, ldo, n1, n2)
  if (dtype == EB_F32) EB_GATE(float);
  else if (dtype == EB_F16) EB_GATE(__half);
  else EB_GATE(__nv_bfloat16);
#undef EB_GATE
  return check_launch("sigmoid_gate");
}
