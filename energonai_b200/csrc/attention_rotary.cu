// What lies between the projection of an attention layer and the attention itself where every head is
// normalised by itself and turned by rotary positions, and the values are the keys as projected:
// queries and keys are divided by their head's root mean square and weighted, neighbouring pairs of the
// first dimensions are rotated by position * frequency, and keys (rotated) and values (as projected) go
// to a ring cache.  Statistics, angles and rotations are fp32 (accurate sine and cosine).
#include "common.cuh"

namespace eb {
namespace {

struct RotaryParams {
  const void *proj;            // rows [q: heads*dk | k: kv_heads*dk]
  long long ldp;
  int heads, kv_heads, dk;
  const void *wq, *wk;         // [dk], zero where padded
  float inv_count, eps;
  const float *freq;           // [pairs]
  int pairs;
  void *q, *k;                 // rows; k may be null
  long long ldq, ldk;
  void *k_cache, *v_cache;
  long long k_bs, k_rs, v_bs, v_rs;
  int ring_rows, rows_per_batch;
  const int *pos_dev, *first;
};

template <typename T> struct Pair;
template <> struct Pair<float> {
  using R = float2;
  static __device__ __forceinline__ float2 get(R r) { return r; }
  static __device__ __forceinline__ R put(float a, float b) { return make_float2(a, b); }
};
template <typename T> struct Pair {
  using R = uint32_t;
  static __device__ __forceinline__ float2 get(R r) { return unpack2<T>(r); }
  static __device__ __forceinline__ R put(float a, float b) { return pack2<T>(a, b); }
};

// One row per CTA, a head per warp at a time; lane l has the pairs l, l + 32, ... of a head.
template <typename T, int PAIRS>
__global__ void attention_rotary_kernel(const RotaryParams p) {
  using P = Pair<T>;
  using R = typename P::R;
  griddep_wait();
  griddep_launch();
  const long long row = blockIdx.x, b = row / p.rows_per_batch;
  const int s = (int)(row - b * p.rows_per_batch), col = (p.pos_dev ? *p.pos_dev : 0) + s;
  const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = p.dk / 2, all = p.heads + p.kv_heads;
  const bool keep = col >= 0 && p.rows_per_batch - s <= p.ring_rows;
  const long long ring = col >= 0 ? col % p.ring_rows : 0;
  const R *x = reinterpret_cast<const R *>(reinterpret_cast<const T *>(p.proj) + row * p.ldp);
  R *q = reinterpret_cast<R *>(reinterpret_cast<T *>(p.q) + row * p.ldq);
  R *k = p.k ? reinterpret_cast<R *>(reinterpret_cast<T *>(p.k) + row * p.ldk) : nullptr;
  R *kc = reinterpret_cast<R *>(reinterpret_cast<T *>(p.k_cache) + b * p.k_bs + ring * p.k_rs);
  R *vc = reinterpret_cast<R *>(reinterpret_cast<T *>(p.v_cache) + b * p.v_bs + ring * p.v_rs);
  const float at = (float)max(0, col - (p.first ? p.first[b] : 0));
  float cs[PAIRS], sn[PAIRS];
#pragma unroll
  for (int i = 0; i < PAIRS; ++i) {
    const int c = lane + 32 * i;
    cs[i] = 1.f;
    sn[i] = 0.f;
    if (c < p.pairs) sincosf(at * p.freq[c], &sn[i], &cs[i]);
  }
  for (int h = warp; h < all; h += warps) {
    const bool is_k = h >= p.heads;
    const R *w = reinterpret_cast<const R *>(is_k ? p.wk : p.wq);
    R raw[PAIRS];
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const int c = lane + 32 * i;
      if (c >= half) break;
      raw[i] = x[h * half + c];
      const float2 f = P::get(raw[i]);
      sq = fmaf(f.x, f.x, fmaf(f.y, f.y, sq));
    }
    const float r = 1.f / sqrtf(warp_sum(sq) * p.inv_count + p.eps);
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const int c = lane + 32 * i;
      if (c >= half) break;
      const float2 f = P::get(raw[i]), wv = P::get(w[c]);
      const float u = f.x * r * wv.x, v = f.y * r * wv.y;
      const R y = P::put(u * cs[i] - v * sn[i], v * cs[i] + u * sn[i]);
      if (!is_k) {
        q[h * half + c] = y;
      } else {
        const int at_k = (h - p.heads) * half + c;
        if (k) k[at_k] = y;
        if (keep) {
          kc[at_k] = y;
          vc[at_k] = raw[i];
        }
      }
    }
  }
}

template <typename T> int launch_rotary(const RotaryParams &p, int n1, cudaStream_t st) {
  const int all = p.heads + p.kv_heads, need = (p.dk / 2 + 31) / 32;
  const int most = n1 >= 4 * sm_count() ? 8 : 16;           // few rows: fewer heads one after the other
  const dim3 g(n1), b(32 * (all < most ? all : most));
  if (need <= 1) launch_pdl(attention_rotary_kernel<T, 1>, g, b, 0, st, p);
  else if (need <= 2) launch_pdl(attention_rotary_kernel<T, 2>, g, b, 0, st, p);
  else if (need <= 4) launch_pdl(attention_rotary_kernel<T, 4>, g, b, 0, st, p);
  else if (need <= 16) launch_pdl(attention_rotary_kernel<T, 16>, g, b, 0, st, p);
  else return fail(EB_EUNSUPPORTED, "attention_rotary: head size %d is too large (1024)", p.dk);
  return check_launch("attention_rotary");
}

}  // namespace
}  // namespace eb

using namespace eb;

extern "C" int eb_attention_rotary(const void *proj, long long ldp, int heads, int kv_heads, int dk, int dk_count, const void *q_norm,
                                   const void *k_norm, float eps, const float *freq, int pairs, void *q_out, long long ldq, void *k_out,
                                   long long ldk, void *k_cache, long long k_batch_stride, long long k_row_stride, void *v_cache,
                                   long long v_batch_stride, long long v_row_stride, int ring_rows, int n1, int rows_per_batch,
                                   const int32_t *pos_device, const int32_t *first, int dtype, void *stream) {
  if (n1 == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "attention_rotary: bad dtype %d", dtype);
  EB_REQUIRE(proj && q_norm && k_norm && q_out && k_cache && v_cache, "attention_rotary: null pointer");
  EB_REQUIRE(heads > 0 && kv_heads > 0 && dk > 0 && dk % 8 == 0 && (long long)(heads + kv_heads) * dk < (1 << 28), "attention_rotary: head sizes must be multiples of 8 (%d)", dk);
  EB_REQUIRE(dk_count > 0 && dk_count <= dk && pairs >= 0 && 2 * pairs <= dk_count && (pairs == 0 || freq), "attention_rotary: at most half of the dimensions are pairs");
  EB_REQUIRE(n1 > 0 && rows_per_batch > 0 && n1 % rows_per_batch == 0 && ring_rows > 0, "attention_rotary: bad row counts");
  const long long strides[] = {ldp, ldq, k_out ? ldk : 0, k_batch_stride, k_row_stride, v_batch_stride, v_row_stride};
  for (long long s : strides) EB_REQUIRE(s % 8 == 0, "attention_rotary: strides must be multiples of 8 elements");
  EB_REQUIRE(ldp >= (long long)(heads + kv_heads) * dk && ldq >= (long long)heads * dk && (!k_out || ldk >= (long long)kv_heads * dk) &&
                 k_row_stride >= (long long)kv_heads * dk && v_row_stride >= (long long)kv_heads * dk, "attention_rotary: row strides smaller than the rows they hold");
  EB_REQUIRE(aligned16(proj) && aligned16(q_norm) && aligned16(k_norm) && aligned16(q_out) && aligned16(k_out) && aligned16(k_cache) && aligned16(v_cache),
             "attention_rotary: pointers must be 16-byte aligned");
  RotaryParams p{};
  p.proj = proj; p.ldp = ldp; p.heads = heads; p.kv_heads = kv_heads; p.dk = dk; p.wq = q_norm; p.wk = k_norm; p.inv_count = 1.f / (float)dk_count;
  p.eps = eps; p.freq = freq; p.pairs = pairs; p.q = q_out; p.ldq = ldq; p.k = k_out; p.ldk = ldk; p.k_cache = k_cache; p.k_bs = k_batch_stride;
  p.k_rs = k_row_stride; p.v_cache = v_cache; p.v_bs = v_batch_stride; p.v_rs = v_row_stride; p.ring_rows = ring_rows; p.rows_per_batch = rows_per_batch;
  p.pos_dev = pos_device; p.first = first;
  cudaStream_t st = as_stream(stream);
  if (dtype == EB_F32) return launch_rotary<float>(p, n1, st);
  if (dtype == EB_F16) return launch_rotary<__half>(p, n1, st);
  return launch_rotary<__nv_bfloat16>(p, n1, st);
}
