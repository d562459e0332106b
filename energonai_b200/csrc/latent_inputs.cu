// What lies between the projections of a latent-attention layer with rotary positions and the attention itself:
//
//   latent_inputs   a projected row [query latent | key / value latent, shared rotated key part]: the query latent
//                   is normalised for its up-projection; the key / value latent is normalised, the key part
//                   is turned by its position, and both go, as one row, to the cache and (prompts) a buffer.
//   rotate_heads    the rotated columns of every head of a row, turned in place.
//
// Neighbouring pairs turn by position * frequency, sine and cosine times a common factor.  Statistics, angles
// (accurate sine and cosine) and rotations are fp32.
#include "common.cuh"

namespace eb {
namespace {

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

struct LatentInParams {
  const void *proj;            // rows [q latent: q_cols | c: rot_col | rotated part ... : row_cols - rot_col]
  long long ldp;
  int q_cols, row_cols, rot_col, pairs;
  const void *wq, *wc;         // [q_cols], [rot_col]; zero where padded
  float q_inv, c_inv, eps;
  const float *freq;
  float factor;
  void *q, *rows;              // [n1][q_cols]; [n1][row_cols] or null
  long long ldq, ldr;
  void *ring;                  // null: the layer has no latents of its own
  long long ring_bs, ring_ld;
  int ring_rows, n1, rows_per_batch;
  const int *pos_dev, *first;
};

// A warp per (row, part): part 0 the query latent, part 1 the cached row.
template <typename T>
__global__ void __launch_bounds__(256) latent_inputs_kernel(const LatentInParams p) {
  using P = Pair<T>;
  using R = typename P::R;
  griddep_wait();
  griddep_launch();
  const int parts = p.ring ? 2 : 1, lane = threadIdx.x & 31;
  const long long unit = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), row = unit / parts;
  if (row >= p.n1) return;
  const bool latent = unit % parts == 1;
  const R *x = reinterpret_cast<const R *>(reinterpret_cast<const T *>(p.proj) + row * p.ldp + (latent ? p.q_cols : 0));
  const R *w = reinterpret_cast<const R *>(latent ? p.wc : p.wq);
  const int n = (latent ? p.rot_col : p.q_cols) / 2;
  float sq = 0.f;
#pragma unroll 4
  for (int i = lane; i < n; i += 32) {
    const float2 f = P::get(x[i]);
    sq = fmaf(f.x, f.x, fmaf(f.y, f.y, sq));
  }
  const float r = 1.f / sqrtf(warp_sum(sq) * (latent ? p.c_inv : p.q_inv) + p.eps);
  if (!latent) {
    R *q = reinterpret_cast<R *>(reinterpret_cast<T *>(p.q) + row * p.ldq);
#pragma unroll 4
    for (int i = lane; i < n; i += 32) {
      const float2 f = P::get(x[i]), wv = P::get(w[i]);
      q[i] = P::put(f.x * r * wv.x, f.y * r * wv.y);
    }
    return;
  }
  const long long b = row / p.rows_per_batch;
  const int s = (int)(row - b * p.rows_per_batch), col = (p.pos_dev ? *p.pos_dev : 0) + s;
  const bool keep = col >= 0 && p.rows_per_batch - s <= p.ring_rows;
  R *ring = reinterpret_cast<R *>(reinterpret_cast<T *>(p.ring) + b * p.ring_bs + (keep ? col % p.ring_rows : 0) * p.ring_ld);
  R *rows = p.rows ? reinterpret_cast<R *>(reinterpret_cast<T *>(p.rows) + row * p.ldr) : nullptr;
  const float at = (float)max(0, col - (p.first ? p.first[b] : 0));
  for (int i = lane; i < p.row_cols / 2; i += 32) {
    const float2 f = P::get(x[i]);
    R y;
    if (i < n) {
      const float2 wv = P::get(w[i]);
      y = P::put(f.x * r * wv.x, f.y * r * wv.y);
    } else {
      float sn = 0.f, cs = 0.f;                    // (columns behind the rotated part are padding: zero)
      if (i - n < p.pairs) sincosf(at * p.freq[i - n], &sn, &cs);
      sn *= p.factor;
      cs *= p.factor;
      y = P::put(f.x * cs - f.y * sn, f.y * cs + f.x * sn);
    }
    if (rows) rows[i] = y;
    if (keep) ring[i] = y;
  }
}

struct RotateParams {
  void *x;
  long long ldx;
  int heads, head_cols, col, pairs, rows_per_batch;
  const float *freq;
  float factor;
  const int *pos_dev, *first;
};

template <typename T>
__global__ void __launch_bounds__(512) rotate_heads_kernel(const RotateParams p) {
  using P = Pair<T>;
  using R = typename P::R;
  extern __shared__ float2 cs[];                   // [pairs]
  griddep_wait();
  griddep_launch();
  const long long row = blockIdx.x, b = row / p.rows_per_batch;
  const int col = (p.pos_dev ? *p.pos_dev : 0) + (int)(row - b * p.rows_per_batch);
  const float at = (float)max(0, col - (p.first ? p.first[b] : 0));
  for (int i = threadIdx.x; i < p.pairs; i += blockDim.x) {
    float s, c;
    sincosf(at * p.freq[i], &s, &c);
    cs[i] = make_float2(c * p.factor, s * p.factor);
  }
  __syncthreads();
  R *x = reinterpret_cast<R *>(reinterpret_cast<T *>(p.x) + row * p.ldx + p.col);
#pragma unroll 4
  for (int i = threadIdx.x; i < p.heads * p.pairs; i += blockDim.x) {
    const int h = i / p.pairs, k = i - h * p.pairs;
    R *at_x = x + (long long)h * (p.head_cols / 2) + k;
    const float2 f = P::get(*at_x), t = cs[k];
    *at_x = P::put(f.x * t.x - f.y * t.y, f.y * t.x + f.x * t.y);
  }
}

}  // namespace
}  // namespace eb

using namespace eb;

extern "C" int eb_latent_inputs(const void *proj, long long ldp, int q_cols, int q_count, const void *q_norm, void *q_out, long long ldq,
                                int row_cols, int rot_col, int c_count, const void *c_norm, int pairs, const float *freq, float factor, float eps,
                                void *rows_out, long long ldr, void *ring, long long ring_batch_stride, long long ring_ld, int ring_rows, int n1,
                                int rows_per_batch, const int32_t *pos_device, const int32_t *first, int dtype, void *stream) {
  if (n1 == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "latent_inputs: bad dtype %d", dtype);
  EB_REQUIRE(proj && q_norm && q_out && (!ring || (c_norm && (pairs == 0 || freq))), "latent_inputs: null pointer");
  EB_REQUIRE(n1 > 0 && rows_per_batch > 0 && n1 % rows_per_batch == 0, "latent_inputs: bad row counts");
  EB_REQUIRE(q_cols > 0 && q_cols % 8 == 0 && q_count > 0 && q_count <= q_cols && ldq >= q_cols && ldq % 2 == 0, "latent_inputs: the query latent has %d columns", q_cols);
  EB_REQUIRE(ldp >= q_cols + (ring ? row_cols : 0) && ldp % 2 == 0, "latent_inputs: row strides smaller than the rows they hold");
  EB_REQUIRE(!rows_out || ring, "latent_inputs: rows without a cache");
  if (ring) {
    EB_REQUIRE(rot_col > 0 && rot_col % 2 == 0 && c_count > 0 && c_count <= rot_col && row_cols % 8 == 0 && pairs >= 0 && rot_col + 2 * pairs <= row_cols,
               "latent_inputs: a row of %d columns, the rotated part from %d on", row_cols, rot_col);
    EB_REQUIRE(ring_rows > 0 && ring_ld >= row_cols && ring_ld % 2 == 0 && ring_batch_stride % 2 == 0 && (!rows_out || (ldr >= row_cols && ldr % 2 == 0)),
               "latent_inputs: row strides smaller than the rows they hold");
  }
  EB_REQUIRE(aligned16(proj) && aligned16(q_norm) && aligned16(q_out) && aligned16(c_norm) && aligned16(rows_out) && aligned16(ring),
             "latent_inputs: pointers must be 16-byte aligned");
  LatentInParams p{};
  p.proj = proj; p.ldp = ldp; p.q_cols = q_cols; p.row_cols = row_cols; p.rot_col = rot_col; p.pairs = pairs; p.wq = q_norm; p.wc = c_norm;
  p.q_inv = 1.f / (float)q_count; p.c_inv = ring ? 1.f / (float)c_count : 0.f; p.eps = eps; p.freq = freq; p.factor = factor; p.q = q_out; p.ldq = ldq;
  p.rows = rows_out; p.ldr = ldr; p.ring = ring; p.ring_bs = ring_batch_stride; p.ring_ld = ring_ld; p.ring_rows = ring_rows; p.n1 = n1;
  p.rows_per_batch = rows_per_batch; p.pos_dev = pos_device; p.first = first;
  cudaStream_t st = as_stream(stream);
  const long long warps = (long long)n1 * (ring ? 2 : 1), per = warps < 8ll * sm_count() ? 1 : 8;     // few rows: a warp per CTA
  const dim3 g((unsigned)((warps + per - 1) / per)), t((unsigned)(32 * per));
  if (dtype == EB_F32) launch_pdl(latent_inputs_kernel<float>, g, t, 0, st, p);
  else if (dtype == EB_F16) launch_pdl(latent_inputs_kernel<__half>, g, t, 0, st, p);
  else launch_pdl(latent_inputs_kernel<__nv_bfloat16>, g, t, 0, st, p);
  return check_launch("latent_inputs");
}

extern "C" int eb_rotate_heads(void *x, long long ldx, int heads, int head_cols, int col, int pairs, const float *freq, float factor, int n1,
                               int rows_per_batch, const int32_t *pos_device, const int32_t *first, int dtype, void *stream) {
  if (n1 == 0 || pairs == 0) return EB_OK;
  EB_REQUIRE(dtype_ok(dtype), "rotate_heads: bad dtype %d", dtype);
  EB_REQUIRE(x && freq && aligned16(x), "rotate_heads: null or misaligned pointer");
  EB_REQUIRE(n1 > 0 && rows_per_batch > 0 && n1 % rows_per_batch == 0 && heads > 0, "rotate_heads: bad row counts");
  EB_REQUIRE(head_cols % 2 == 0 && col >= 0 && col % 2 == 0 && pairs > 0 && pairs <= 2048 && col + 2 * pairs <= head_cols && ldx % 2 == 0 &&
                 ldx >= (long long)heads * head_cols, "rotate_heads: %d pairs from column %d of heads of %d", pairs, col, head_cols);
  RotateParams p{};
  p.x = x; p.ldx = ldx; p.heads = heads; p.head_cols = head_cols; p.col = col; p.pairs = pairs; p.rows_per_batch = rows_per_batch;
  p.freq = freq; p.factor = factor; p.pos_dev = pos_device; p.first = first;
  cudaStream_t st = as_stream(stream);
  const size_t smem = (size_t)pairs * sizeof(float2);
  const dim3 t(n1 < 4 * sm_count() && heads * pairs > 256 ? 512 : 128);                    // few rows: fewer pairs one after the other
  if (dtype == EB_F32) launch_pdl(rotate_heads_kernel<float>, dim3(n1), t, smem, st, p);
  else if (dtype == EB_F16) launch_pdl(rotate_heads_kernel<__half>, dim3(n1), t, smem, st, p);
  else launch_pdl(rotate_heads_kernel<__nv_bfloat16>, dim3(n1), t, smem, st, p);
  return check_launch("rotate_heads");
}
