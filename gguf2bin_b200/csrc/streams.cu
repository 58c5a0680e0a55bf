// Several residual streams side by side: X [T, S, H] in 32-bit, S copies of what other models keep one of.
//   read   u = sum_s a_s X_s (a missing: ones), and h = u / sqrt(mean(u^2) + eps) * w in the compute type: what a
//          sublayer reads, or with ones the sum in front of the head
//   join   X'_t = sum_s mix[s, t] X_s + m out[t] y, all streams at once from the old ones (y: the sublayer's result),
//          and in the same pass h of the next sublayer from the new streams: u = sum_t a_t X'_t, normed
// S = 1 with mix = out = a = 1 is the ordinary x += m y with the next norm.  Coefficients, sums and norms are 32-bit.
#include "common.cuh"

G2B_DEFINE_LAST_ERROR

#define STREAMS_MAX 16

struct StreamsNext {                  // the reader behind a join
  const float *in;                    // [S] or null: ones
  const float *w;                     // [H] or null: ones
  float eps;
  void *h;                            // [T, H] in the compute type, or null: no reader
};

__device__ __forceinline__ void store4(float *p, const float4 &v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void store4(bf16 *p, const float4 &v) {
  uint2 raw;
  *reinterpret_cast<__nv_bfloat162 *>(&raw.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162 *>(&raw.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2 *>(p) = raw;
}
__device__ __forceinline__ float4 fma4(float a, const float4 &x, const float4 &c) {
  return make_float4(fmaf(a, x.x, c.x), fmaf(a, x.y, c.y), fmaf(a, x.z, c.z), fmaf(a, x.w, c.w));
}
__device__ __forceinline__ float dot4(const float4 &x, float c) {
  return fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, fmaf(x.w, x.w, c))));
}

// A block a row; a thread keeps PER groups of four neighbours of every stream in registers.  JOIN false: nothing is
// written back, `rows` may gather rows.
// (No __restrict__ on what earlier kernels write: the compiler may move loads through such pointers above pdl_wait().)
template <typename T, int S, int PER, bool JOIN>
__global__ void __launch_bounds__(256)
streams_kernel(float *X, const float *y, const float *__restrict__ mix, const float *__restrict__ out, float m, const int *rows,
               const StreamsNext next, int H) {
  __shared__ float scratch[32];
  pdl_launch();
  // coefficients and norm weights are no earlier kernel's output
  float A[S], M[JOIN ? S * S : 1], O[S];
#pragma unroll
  for (int s = 0; s < S; ++s) A[s] = next.in ? __ldg(next.in + s) : 1.f;
  if (JOIN) {
#pragma unroll
    for (int i = 0; i < S * S; ++i) M[JOIN ? i : 0] = __ldg(mix + i);
#pragma unroll
    for (int s = 0; s < S; ++s) O[s] = m * __ldg(out + s);
  }
  const int r = blockIdx.x, H4 = H >> 2;
  float4 w[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int j = threadIdx.x + blockDim.x * i;
    w[i] = next.w && j < H4 ? *reinterpret_cast<const float4 *>(next.w + 4 * j) : make_float4(1.f, 1.f, 1.f, 1.f);
  }
  pdl_wait();
  const int t = rows ? rows[r] : r;
  float *xr = X + (size_t)t * S * H;
  float4 u[PER];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int j = threadIdx.x + blockDim.x * i;
    if (j >= H4) continue;
    float4 x[S];
#pragma unroll
    for (int s = 0; s < S; ++s) x[s] = *reinterpret_cast<const float4 *>(xr + (size_t)s * H + 4 * j);
    u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (JOIN) {
      const float4 yv = *reinterpret_cast<const float4 *>(y + (size_t)t * H + 4 * j);
#pragma unroll
      for (int d = 0; d < S; ++d) {
        float4 v = make_float4(O[d] * yv.x, O[d] * yv.y, O[d] * yv.z, O[d] * yv.w);
#pragma unroll
        for (int s = 0; s < S; ++s) v = fma4(M[JOIN ? s * S + d : 0], x[s], v);
        *reinterpret_cast<float4 *>(xr + (size_t)d * H + 4 * j) = v;
        u[i] = fma4(A[d], v, u[i]);
      }
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s) u[i] = fma4(A[s], x[s], u[i]);
    }
    ss = dot4(u[i], ss);
  }
  if (!next.h) return;
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)H + next.eps);
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int j = threadIdx.x + blockDim.x * i;
    if (j >= H4) continue;
    store4((T *)next.h + (size_t)r * H + 4 * j,
           make_float4((w[i].x * u[i].x) * inv, (w[i].y * u[i].y) * inv, (w[i].z * u[i].z) * inv, (w[i].w * u[i].w) * inv));
  }
}

// Any number of streams up to STREAMS_MAX, any width: an element at a time, u once more from what the thread wrote.
template <typename T, bool JOIN>
__global__ void __launch_bounds__(256)
streams_any_kernel(float *__restrict__ X, const float *__restrict__ y, const float *__restrict__ mix,
                   const float *__restrict__ out, float m, const int *__restrict__ rows, const StreamsNext next, int S, int H) {
  __shared__ float scratch[32], A[STREAMS_MAX], M[STREAMS_MAX * STREAMS_MAX], O[STREAMS_MAX];
  pdl_launch();
  pdl_wait();
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    A[i] = next.in ? next.in[i] : 1.f;
    if (JOIN) O[i] = m * out[i];
  }
  if (JOIN)
    for (int i = threadIdx.x; i < S * S; i += blockDim.x) M[i] = mix[i];
  __syncthreads();
  const int r = blockIdx.x, t = rows ? rows[r] : r;
  float *xr = X + (size_t)t * S * H;
  float ss = 0.f;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    float u = 0.f;
    if (JOIN) {
      float x[STREAMS_MAX];
#pragma unroll
      for (int s = 0; s < STREAMS_MAX; ++s) x[s] = s < S ? xr[(size_t)s * H + j] : 0.f;
      const float yv = y[(size_t)t * H + j];
      for (int d = 0; d < S; ++d) {
        float v = O[d] * yv;
#pragma unroll
        for (int s = 0; s < STREAMS_MAX; ++s)
          if (s < S) v = fmaf(M[s * S + d], x[s], v);
        xr[(size_t)d * H + j] = v;
        u = fmaf(A[d], v, u);
      }
    } else {
      for (int s = 0; s < S; ++s) u = fmaf(A[s], xr[(size_t)s * H + j], u);
    }
    ss = fmaf(u, u, ss);
  }
  if (!next.h) return;
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)H + next.eps);
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    float u = 0.f;
    for (int s = 0; s < S; ++s) u = fmaf(A[s], xr[(size_t)s * H + j], u);
    ((T *)next.h)[(size_t)r * H + j] = from_f32<T>(((next.w ? next.w[j] : 1.f) * u) * inv);
  }
}

template <typename T, int S, bool JOIN>
static bool launch_fixed(float *X, const float *y, const float *mix, const float *out, float m, const int *rows, int n_rows,
                         const StreamsNext &next, int H, cudaStream_t stream) {
  const int H4 = H >> 2;
  int threads = (H4 + 31) / 32 * 32;
  threads = threads > 256 ? 256 : threads;
#define STREAMS_CASE(PER_)                                                                                                   \
  if (H4 <= (PER_) * 256) {                                                                                                  \
    g2b_launch(streams_kernel<T, S, PER_, JOIN>, dim3(n_rows), dim3(threads), 0, stream, X, y, mix, out, m, rows, next, H);  \
    return true;                                                                                                             \
  }
  STREAMS_CASE(1) STREAMS_CASE(2) STREAMS_CASE(4) STREAMS_CASE(8)
#undef STREAMS_CASE
  return false;
}

template <typename T, bool JOIN>
static void launch_streams(float *X, const float *y, const float *mix, const float *out, float m, const int *rows, int n_rows,
                           const StreamsNext &next, int S, int H, cudaStream_t stream) {
  const bool aligned = H % 4 == 0 && !(((uintptr_t)X | (uintptr_t)y | (uintptr_t)next.w | (uintptr_t)next.h) & 15);
  bool done = false;
  if (aligned) {
    if (S == 1) done = launch_fixed<T, 1, JOIN>(X, y, mix, out, m, rows, n_rows, next, H, stream);
    else if (S == 2) done = launch_fixed<T, 2, JOIN>(X, y, mix, out, m, rows, n_rows, next, H, stream);
    else if (S == 3) done = launch_fixed<T, 3, JOIN>(X, y, mix, out, m, rows, n_rows, next, H, stream);
    else if (S == 4) done = launch_fixed<T, 4, JOIN>(X, y, mix, out, m, rows, n_rows, next, H, stream);
  }
  if (!done)
    g2b_launch(streams_any_kernel<T, JOIN>, dim3(n_rows), dim3(256), 0, stream, X, y, mix, out, m, rows, next, S, H);
}

// X [T, S, H]; h [n_rows, H]; rows (int32 [n_rows]) gathers tokens, null: 0 .. n_rows - 1
extern "C" int g2b_streams_read(const float *X, const float *in, const float *w, float eps, const int *rows, int n_rows, int S,
                                int H, void *h, int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (S < 1 || S > STREAMS_MAX || H <= 0) G2B_REFUSE("streams_read: %d streams (1..%d) of %d", S, STREAMS_MAX, H);
  const StreamsNext next = {in, w, eps, h};
  if (dtype == G2B_F32)
    launch_streams<float, false>((float *)X, nullptr, nullptr, nullptr, 0.f, rows, n_rows, next, S, H, stream);
  else if (dtype == G2B_BF16)
    launch_streams<bf16, false>((float *)X, nullptr, nullptr, nullptr, 0.f, rows, n_rows, next, S, H, stream);
  else
    G2B_REFUSE("streams_read: unknown dtype %d", dtype);
  return g2b_check_launch("streams_read");
}

// mix [S from, S to], out [S]; h null: no reader behind the join
extern "C" int g2b_streams_join(float *X, const float *y, const float *mix, const float *out, float m, int T_tokens, int S, int H,
                                const float *in, const float *w, float eps, void *h, int dtype, cudaStream_t stream) {
  if (T_tokens <= 0) return 0;
  if (S < 1 || S > STREAMS_MAX || H <= 0) G2B_REFUSE("streams_join: %d streams (1..%d) of %d", S, STREAMS_MAX, H);
  if (!y || !mix || !out) G2B_REFUSE("streams_join: a result and its coefficients are needed");
  const StreamsNext next = {in, w, eps, h};
  if (dtype == G2B_F32)
    launch_streams<float, true>(X, y, mix, out, m, nullptr, T_tokens, next, S, H, stream);
  else if (dtype == G2B_BF16)
    launch_streams<bf16, true>(X, y, mix, out, m, nullptr, T_tokens, next, S, H, stream);
  else
    G2B_REFUSE("streams_join: unknown dtype %d", dtype);
  return g2b_check_launch("streams_join");
}
