// How a sublayer's result joins the stream in a layer that norms it on the way in and on the way out:
//   x <- x + y / sqrt(mean(y^2) + eps) * w  (+ add),  then  next = x / sqrt(mean(x^2) + next_eps) * next_w
// in one pass over the row: the new stream in 32-bit and the next sublayer's input in the compute type.  Where
// y comes from is a functor: a row of a buffer, or a routed feed-forward's weighted sum of its experts' rows.
// `add` (a row of another 32-bit buffer) is what a model adds to its stream between two layers.
#pragma once
#include "common.cuh"

struct JoinTail {
  const float *w;             // [H] the result's norm weight (null: ones)
  float eps;
  const float *add;           // [T, H] or null
  const float *next_w;        // [H] the next norm's weight (null: ones)
  float next_eps;
  void *next;                 // [T, H] in the compute type, or null: no next norm
};

struct JoinRow {              // y as it lies in a buffer
  const float *y;
  __device__ __forceinline__ float4 four(int t, int H, int j, const float4 &) const {
    return *reinterpret_cast<const float4 *>(y + (size_t)t * H + j);
  }
  __device__ __forceinline__ float one(int t, int H, int j, float) const { return y[(size_t)t * H + j]; }
};

struct JoinExperts {          // y = base + sum_r weight_r * (row of the pair, or the token's own input where it has none)
  const float *rows;
  const int *pair_row;
  const float *weight;
  const float *base;          // [T, H] or null
  int top;
  __device__ __forceinline__ float4 four(int t, int H, int j, const float4 &own) const {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int r = 0; r < top; ++r) {
      const int row = pair_row[(size_t)t * top + r];
      const float wt = weight[(size_t)t * top + r];
      const float4 v = row >= 0 ? *reinterpret_cast<const float4 *>(rows + (size_t)row * H + j) : own;
      a.x = fmaf(wt, v.x, a.x), a.y = fmaf(wt, v.y, a.y), a.z = fmaf(wt, v.z, a.z), a.w = fmaf(wt, v.w, a.w);
    }
    if (base) {
      const float4 b = *reinterpret_cast<const float4 *>(base + (size_t)t * H + j);
      a.x += b.x, a.y += b.y, a.z += b.z, a.w += b.w;
    }
    return a;
  }
  __device__ __forceinline__ float one(int t, int H, int j, float own) const {
    float a = 0.f;
    for (int r = 0; r < top; ++r) {
      const int row = pair_row[(size_t)t * top + r];
      a = fmaf(weight[(size_t)t * top + r], row >= 0 ? rows[(size_t)row * H + j] : own, a);
    }
    return base ? a + base[(size_t)t * H + j] : a;
  }
};

__device__ __forceinline__ void join_store4(float *p, const float4 &v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void join_store4(bf16 *p, const float4 &v) {
  uint2 raw;
  *reinterpret_cast<__nv_bfloat162 *>(&raw.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162 *>(&raw.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2 *>(p) = raw;
}

// A block a row; a thread keeps PER groups of four neighbours of y and of x in registers.
template <typename T, int PER, typename Y>
__global__ void __launch_bounds__(256)
join_norm_kernel(float *__restrict__ x, const Y from, const JoinTail a, int H) {
  pdl_launch();
  pdl_wait();
  __shared__ float scratch[32];
  const int t = blockIdx.x, H4 = H >> 2;
  float *xr = x + (size_t)t * H;
  float4 y[PER], s[PER];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int j = threadIdx.x + blockDim.x * i;
    if (j < H4) {
      s[i] = *reinterpret_cast<const float4 *>(xr + 4 * j);
      y[i] = from.four(t, H, 4 * j, s[i]);
      ss = fmaf(y[i].x, y[i].x, fmaf(y[i].y, y[i].y, fmaf(y[i].z, y[i].z, fmaf(y[i].w, y[i].w, ss))));
    }
  }
  ss = block_sum(ss, scratch);
  const float inv = 1.f / sqrtf(ss / (float)H + a.eps);
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int j = threadIdx.x + blockDim.x * i;
    if (j < H4) {
      const float4 w = a.w ? *reinterpret_cast<const float4 *>(a.w + 4 * j) : make_float4(1.f, 1.f, 1.f, 1.f);
      s[i].x += (y[i].x * inv) * w.x, s[i].y += (y[i].y * inv) * w.y;
      s[i].z += (y[i].z * inv) * w.z, s[i].w += (y[i].w * inv) * w.w;
      if (a.add) {
        const float4 e = *reinterpret_cast<const float4 *>(a.add + (size_t)t * H + 4 * j);
        s[i].x += e.x, s[i].y += e.y, s[i].z += e.z, s[i].w += e.w;
      }
      *reinterpret_cast<float4 *>(xr + 4 * j) = s[i];
      ss = fmaf(s[i].x, s[i].x, fmaf(s[i].y, s[i].y, fmaf(s[i].z, s[i].z, fmaf(s[i].w, s[i].w, ss))));
    }
  }
  if (!a.next) return;
  ss = block_sum(ss, scratch);
  const float ninv = 1.f / sqrtf(ss / (float)H + a.next_eps);
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int j = threadIdx.x + blockDim.x * i;
    if (j < H4) {
      const float4 w = a.next_w ? *reinterpret_cast<const float4 *>(a.next_w + 4 * j) : make_float4(1.f, 1.f, 1.f, 1.f);
      join_store4((T *)a.next + (size_t)t * H + 4 * j,
                  make_float4((w.x * s[i].x) * ninv, (w.y * s[i].y) * ninv, (w.z * s[i].z) * ninv, (w.w * s[i].w) * ninv));
    }
  }
}

// Any row: nothing is kept in registers, an element at a time.
template <typename T, typename Y>
__global__ void __launch_bounds__(256)
join_norm_any_kernel(float *__restrict__ x, const Y from, const JoinTail a, int H) {
  pdl_launch();
  pdl_wait();
  __shared__ float scratch[32];
  const int t = blockIdx.x;
  float *xr = x + (size_t)t * H;
  float ss = 0.f;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    const float v = from.one(t, H, j, xr[j]);
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, scratch);
  const float inv = 1.f / sqrtf(ss / (float)H + a.eps);
  ss = 0.f;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    const float own = xr[j];
    float v = own + (from.one(t, H, j, own) * inv) * (a.w ? a.w[j] : 1.f);
    if (a.add) v += a.add[(size_t)t * H + j];
    xr[j] = v;
    ss = fmaf(v, v, ss);
  }
  if (!a.next) return;
  ss = block_sum(ss, scratch);
  const float ninv = 1.f / sqrtf(ss / (float)H + a.next_eps);
  for (int j = threadIdx.x; j < H; j += blockDim.x)
    ((T *)a.next)[(size_t)t * H + j] = from_f32<T>(((a.next_w ? a.next_w[j] : 1.f) * xr[j]) * ninv);
}

template <typename T, typename Y>
static void launch_join(float *x, const Y &from, const JoinTail &a, int n_rows, int H, bool aligned, cudaStream_t stream) {
  const int H4 = H >> 2;
  int threads = (H4 + 31) / 32 * 32;
  threads = threads > 256 ? 256 : threads;
  if (!aligned || (H & 3) || H4 > 8 * 256)
    g2b_launch(join_norm_any_kernel<T, Y>, dim3(n_rows), dim3(256), 0, stream, x, from, a, H);
  else if (H4 <= 256)
    g2b_launch(join_norm_kernel<T, 1, Y>, dim3(n_rows), dim3(threads), 0, stream, x, from, a, H);
  else if (H4 <= 512)
    g2b_launch(join_norm_kernel<T, 2, Y>, dim3(n_rows), dim3(256), 0, stream, x, from, a, H);
  else if (H4 <= 1024)
    g2b_launch(join_norm_kernel<T, 4, Y>, dim3(n_rows), dim3(256), 0, stream, x, from, a, H);
  else
    g2b_launch(join_norm_kernel<T, 8, Y>, dim3(n_rows), dim3(256), 0, stream, x, from, a, H);
}
