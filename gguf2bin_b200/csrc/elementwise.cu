// Memory-bound kernels of the step: embedding rows, RMSNorm (optionally on gathered
// rows), fused per-head RMSNorm + half-split rotation + cache write, the cache write
// alone, and the SiLU gate.  All statistics, angles and products are 32-bit.
//
// Formulas (paths relative to AnonymoDGH/gguf2bin):
//   embedding      src/l5_model.c:488-491
//   rmsnorm        src/l3_math.c:34-36,49      o_j = (w_j * x_j) * 1/sqrt(sum x^2 / n + eps)
//   per-head norm  src/l3_math.c:107-114
//   rotation       src/l3_math.c:84-102        pairs (j, j+half), ang = pos * freq_j
//   cache write    src/l5_model.c:232-247      K after norm and rotation, V raw
//   SiLU gate      src/l3_math.c:57-62, src/l5_model.c:594-595
#include "common.cuh"
#include "glu.cuh"

G2B_DEFINE_LAST_ERROR

// E neighbours (4 or 8, a multiple of 4 in float) in accesses of 8 or 16 bytes
template <int E> __device__ __forceinline__ void ldE(const bf16 *p, float (&v)[E]) {
  if constexpr (E == 8) {
    const uint4 raw = *reinterpret_cast<const uint4 *>(p);
    const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&w[i]));
      v[2 * i] = f.x; v[2 * i + 1] = f.y;
    }
  } else {
    const uint2 raw = *reinterpret_cast<const uint2 *>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&raw.y));
    v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
  }
}
template <int E> __device__ __forceinline__ void ldE(const float *p, float (&v)[E]) {
#pragma unroll
  for (int i = 0; i < E; i += 4) {
    const float4 raw = *reinterpret_cast<const float4 *>(p + i);
    v[i] = raw.x; v[i + 1] = raw.y; v[i + 2] = raw.z; v[i + 3] = raw.w;
  }
}
template <int E> __device__ __forceinline__ void stE(bf16 *p, const float (&v)[E]) {
  uint32_t w[E / 2];
#pragma unroll
  for (int i = 0; i < E / 2; ++i) {
    __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    w[i] = *reinterpret_cast<uint32_t *>(&h);
  }
  if constexpr (E == 8) *reinterpret_cast<uint4 *>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  else *reinterpret_cast<uint2 *>(p) = make_uint2(w[0], w[1]);
}
template <int E> __device__ __forceinline__ void stE(float *p, const float (&v)[E]) {
#pragma unroll
  for (int i = 0; i < E; i += 4) *reinterpret_cast<float4 *>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
}

// ---------------------------------------------------------------------------
// embedding: out[t, :] = table[ids[t], :] * scale   (out is the 32-bit residual stream); with a position
// table also + positions[tok_pos[t], :], and a second copy of the rows into `again` when it is given
// ---------------------------------------------------------------------------
template <typename TW>
__global__ void embed_rows_kernel(const TW *__restrict__ table, const int *__restrict__ ids,
                                  float *__restrict__ out, int H, int V, float scale,
                                  const TW *__restrict__ positions, const int *__restrict__ tok_pos, int n_pos,
                                  float *__restrict__ again) {
  pdl_launch();
  pdl_wait();
  const int t = blockIdx.x;
  int id = ids[t];
  const bool ok = (id >= 0 && id < V);
  if (!ok) id = 0;                                   // host validates ids; never read outside
  const TW *row = table + (size_t)id * H;
  float *o = out + (size_t)t * H;
  // rows that only fill a step up may count past the table: their results are never used
  const TW *prow = positions ? positions + (size_t)min(max(tok_pos[t], 0), n_pos - 1) * H : nullptr;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    float v = ok ? to_f32(row[j]) * scale : 0.f;
    if (prow) v += to_f32(prow[j]);
    o[j] = v;
    if (again) again[(size_t)t * H + j] = v;
  }
}

extern "C" int g2b_embed_rows(const void *table, int table_dtype, const int *ids, float *out,
                              int T, int H, int V, float scale, const void *positions, const int *tok_pos,
                              int n_pos, float *again, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (positions && (!tok_pos || n_pos <= 0)) G2B_REFUSE("embed_rows: a position table needs its length and the tokens' positions");
  if (H <= 0 || V <= 0) G2B_REFUSE("embed_rows: bad sizes H=%d V=%d", H, V);
  const int threads = H >= 256 ? 256 : 64;
  if (table_dtype == G2B_F32)
    g2b_launch(embed_rows_kernel<float>, dim3(T), dim3(threads), 0, stream, (const float *)table, ids, out, H, V, scale,
               (const float *)positions, tok_pos, n_pos, again);
  else if (table_dtype == G2B_BF16)
    g2b_launch(embed_rows_kernel<bf16>, dim3(T), dim3(threads), 0, stream, (const bf16 *)table, ids, out, H, V, scale,
               (const bf16 *)positions, tok_pos, n_pos, again);
  else
    G2B_REFUSE("embed_rows: unknown table dtype %d", table_dtype);
  return g2b_check_launch("embed_rows");
}

// The same rows divided by their root mean square, times w, written `copies` times side by side: out [T, copies, H].
template <typename TW, bool VEC>
__global__ void __launch_bounds__(256)
embed_norm_rows_kernel(const TW *__restrict__ table, const int *__restrict__ ids, const float *__restrict__ w, float eps,
                       float *__restrict__ out, int copies, int H, int V, float scale) {
  pdl_launch();
  pdl_wait();
  __shared__ float scratch[32];
  const int t = blockIdx.x;
  int id = ids[t];
  const bool ok = (id >= 0 && id < V);
  if (!ok) id = 0;                                   // host validates ids; never read outside
  const TW *row = table + (size_t)id * H;
  float ss = 0.f;
  if (VEC) {                                         // H a multiple of four, everything on four entries: 16-byte stores
    for (int j = 4 * threadIdx.x; j < H; j += 4 * blockDim.x) {
      float v[4];
      ldE<4>(row + j, v);
#pragma unroll
      for (int i = 0; i < 4; ++i) ss = fmaf(v[i] * scale, v[i] * scale, ss);
    }
    if (!ok) ss = 0.f;
  } else {
    for (int j = threadIdx.x; j < H; j += blockDim.x) {
      const float v = ok ? to_f32(row[j]) * scale : 0.f;
      ss = fmaf(v, v, ss);
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)H + eps);
  if (VEC) {
    for (int j = 4 * threadIdx.x; j < H; j += 4 * blockDim.x) {
      float v[4], g[4] = {1.f, 1.f, 1.f, 1.f};
      ldE<4>(row + j, v);
      if (w) ldE<4>(w + j, g);
#pragma unroll
      for (int i = 0; i < 4; ++i) v[i] = ((ok ? v[i] * scale : 0.f) * inv) * g[i];
      for (int c = 0; c < copies; ++c)
        *reinterpret_cast<float4 *>(out + ((size_t)t * copies + c) * H + j) = make_float4(v[0], v[1], v[2], v[3]);
    }
  } else {
    for (int j = threadIdx.x; j < H; j += blockDim.x) {
      const float v = ((ok ? to_f32(row[j]) * scale : 0.f) * inv) * (w ? w[j] : 1.f);
      for (int c = 0; c < copies; ++c) out[((size_t)t * copies + c) * H + j] = v;
    }
  }
}

extern "C" int g2b_embed_norm_rows(const void *table, int table_dtype, const int *ids, const float *w, float eps, float *out,
                                   int copies, int T, int H, int V, float scale, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || V <= 0 || copies <= 0) G2B_REFUSE("embed_norm_rows: bad sizes H=%d V=%d copies=%d", H, V, copies);
  const bool vec = H % 4 == 0 && !(((uintptr_t)out | (uintptr_t)w) & 15) && !((uintptr_t)table & (table_dtype == G2B_F32 ? 15 : 7));
  const int threads = H >= 256 ? 256 : 64;
  if (table_dtype == G2B_F32)
    g2b_launch(vec ? embed_norm_rows_kernel<float, true> : embed_norm_rows_kernel<float, false>, dim3(T), dim3(threads), 0, stream, (const float *)table, ids, w, eps, out, copies,
               H, V, scale);
  else if (table_dtype == G2B_BF16)
    g2b_launch(vec ? embed_norm_rows_kernel<bf16, true> : embed_norm_rows_kernel<bf16, false>, dim3(T), dim3(threads), 0, stream, (const bf16 *)table, ids, w, eps, out, copies,
               H, V, scale);
  else
    G2B_REFUSE("embed_norm_rows: unknown table dtype %d", table_dtype);
  return g2b_check_launch("embed_norm_rows");
}

// ---------------------------------------------------------------------------
// rmsnorm over rows of the 32-bit stream; rows == nullptr means rows 0..n_rows-1;
// w == nullptr means no per-channel weight (it was multiplied into the next matrix)
// ---------------------------------------------------------------------------
template <typename TO>
__global__ void rmsnorm_kernel(const float *__restrict__ x, const float *__restrict__ w,
                               const int *__restrict__ rows, TO *__restrict__ out, int H,
                               float eps) {
  pdl_launch();
  pdl_wait();
  __shared__ float scratch[32];
  const int r = blockIdx.x;
  const float *xr = x + (size_t)(rows ? rows[r] : r) * H;
  float ss = 0.f;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    const float v = xr[j];
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, scratch);
  const float inv = 1.f / sqrtf(ss / (float)H + eps);
  TO *o = out + (size_t)r * H;
  for (int j = threadIdx.x; j < H; j += blockDim.x) o[j] = from_f32<TO>(((w ? w[j] : 1.f) * xr[j]) * inv);
}

__device__ __forceinline__ void store4(float *p, float a, float b, float c, float d) {
  *reinterpret_cast<float4 *>(p) = make_float4(a, b, c, d);
}
__device__ __forceinline__ void store4(bf16 *p, float a, float b, float c, float d) {
  uint2 raw;
  *reinterpret_cast<__nv_bfloat162 *>(&raw.x) = __floats2bfloat162_rn(a, b);
  *reinterpret_cast<__nv_bfloat162 *>(&raw.y) = __floats2bfloat162_rn(c, d);
  *reinterpret_cast<uint2 *>(p) = raw;
}

// one warp per row, 16-byte loads, eight of them in flight per lane, four outputs per store; rows
// of up to 1,024 elements stay in registers between the two passes; H a multiple of 4
template <typename TO>
__global__ void __launch_bounds__(128)
rmsnorm_rows_kernel(const float *__restrict__ x, const float *__restrict__ w,
                    const int *__restrict__ rows, TO *__restrict__ out, int n_rows, int H,
                    float eps) {
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int r = blockIdx.x * 4 + (threadIdx.x >> 5);
  if (r >= n_rows) return;
  const float *xr = x + (size_t)(rows ? rows[r] : r) * H;
  float ss = 0.f;
  if (H <= 1024) {
    float4 v[8], g[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int k = lane * 4 + 128 * i;
      v[i] = k < H ? *reinterpret_cast<const float4 *>(xr + k) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int k = lane * 4 + 128 * i;
      g[i] = !w ? make_float4(1.f, 1.f, 1.f, 1.f)
                : (k < H ? *reinterpret_cast<const float4 *>(w + k) : make_float4(0.f, 0.f, 0.f, 0.f));
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss);
      ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss);
    }
    ss = warp_sum(ss);
    const float inv = 1.f / sqrtf(ss / (float)H + eps);
    TO *o = out + (size_t)r * H;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int k = lane * 4 + 128 * i;
      if (k < H)
        store4(o + k, (g[i].x * v[i].x) * inv, (g[i].y * v[i].y) * inv, (g[i].z * v[i].z) * inv,
               (g[i].w * v[i].w) * inv);
    }
    return;
  }
  for (int k0 = lane * 4; k0 < H; k0 += 128 * 8) {
    float4 v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int k = k0 + 128 * i;
      v[i] = k < H ? *reinterpret_cast<const float4 *>(xr + k) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss);
      ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss);
    }
  }
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / (float)H + eps);
  TO *o = out + (size_t)r * H;
  for (int k0 = lane * 4; k0 < H; k0 += 128 * 4) {
    float4 v[4], g[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = k0 + 128 * i;
      if (k < H) {
        v[i] = *reinterpret_cast<const float4 *>(xr + k);
        g[i] = w ? *reinterpret_cast<const float4 *>(w + k) : make_float4(1.f, 1.f, 1.f, 1.f);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = k0 + 128 * i;
      if (k < H)
        store4(o + k, (g[i].x * v[i].x) * inv, (g[i].y * v[i].y) * inv, (g[i].z * v[i].z) * inv,
               (g[i].w * v[i].w) * inv);
    }
  }
}

// one block of 256 threads per row for rows of 1,025 to 8,192 elements: the whole row and its
// weights are fetched at once (up to eight 16-byte loads each per thread) and stay in registers
// between the sum and the output; H a multiple of 4
template <typename TO>
__global__ void __launch_bounds__(256)
rmsnorm_block_kernel(const float *__restrict__ x, const float *__restrict__ w,
                     const int *__restrict__ rows, TO *__restrict__ out, int H, float eps) {
  pdl_launch();
  pdl_wait();
  __shared__ float scratch[32];
  const int r = blockIdx.x;
  const float *xr = x + (size_t)(rows ? rows[r] : r) * H;
  float4 v[8], g[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int k = threadIdx.x * 4 + 1024 * i;
    v[i] = k < H ? *reinterpret_cast<const float4 *>(xr + k) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int k = threadIdx.x * 4 + 1024 * i;
    g[i] = !w ? make_float4(1.f, 1.f, 1.f, 1.f)
              : (k < H ? *reinterpret_cast<const float4 *>(w + k) : make_float4(0.f, 0.f, 0.f, 0.f));
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss);
    ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss);
  }
  ss = block_sum(ss, scratch);
  const float inv = 1.f / sqrtf(ss / (float)H + eps);
  TO *o = out + (size_t)r * H;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int k = threadIdx.x * 4 + 1024 * i;
    if (k < H)
      store4(o + k, (g[i].x * v[i].x) * inv, (g[i].y * v[i].y) * inv, (g[i].z * v[i].z) * inv,
             (g[i].w * v[i].w) * inv);
  }
}

extern "C" int g2b_rmsnorm(const float *x, const float *w, const int *rows, int n_rows, int H,
                           float eps, void *out, int out_dtype, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (H <= 0) G2B_REFUSE("rmsnorm: bad width %d", H);
  if (H % 4 == 0 && H >= 128 && ((((uintptr_t)x) | ((uintptr_t)w) | ((uintptr_t)out)) & 15) == 0 &&
      (out_dtype == G2B_F32 || out_dtype == G2B_BF16)) {
    if (H > 1024 && H <= 8192) {
      if (out_dtype == G2B_F32)
        g2b_launch(rmsnorm_block_kernel<float>, dim3((unsigned)n_rows), dim3(256), 0, stream, x, w, rows, (float *)out, H, eps);
      else
        g2b_launch(rmsnorm_block_kernel<bf16>, dim3((unsigned)n_rows), dim3(256), 0, stream, x, w, rows, (bf16 *)out, H, eps);
      return g2b_check_launch("rmsnorm");
    }
    const unsigned blocks = (unsigned)((n_rows + 3) / 4);
    if (out_dtype == G2B_F32)
      g2b_launch(rmsnorm_rows_kernel<float>, dim3(blocks), dim3(128), 0, stream, x, w, rows, (float *)out, n_rows, H, eps);
    else
      g2b_launch(rmsnorm_rows_kernel<bf16>, dim3(blocks), dim3(128), 0, stream, x, w, rows, (bf16 *)out, n_rows, H, eps);
    return g2b_check_launch("rmsnorm");
  }
  const int threads = H >= 1024 ? 256 : (H >= 256 ? 128 : 32);
  if (out_dtype == G2B_F32)
    g2b_launch(rmsnorm_kernel<float>, dim3(n_rows), dim3(threads), 0, stream, x, w, rows, (float *)out, H, eps);
  else if (out_dtype == G2B_BF16)
    g2b_launch(rmsnorm_kernel<bf16>, dim3(n_rows), dim3(threads), 0, stream, x, w, rows, (bf16 *)out, H, eps);
  else
    G2B_REFUSE("rmsnorm: unknown output dtype %d", out_dtype);
  return g2b_check_launch("rmsnorm");
}

// ---------------------------------------------------------------------------
// per-head norm + rotation + cache write.  One warp per (token, head) of the fused
// projection output qkv[t] = [q heads | k heads | v heads].
//   q heads: norm (if q_w), rotate (if a table is given)  -> q_out[t, h*hd + j]
//   k heads: norm (if k_w), rotate (if a table is given)  -> cache K, or k_out when given
//   v heads: copied                                -> cache V, or v_out when given
// Cache of one layer: [n_pages][2][nkv][page_size][hd]; the page of position p of
// sequence b is page_table[b*P + p/page_size].
// ---------------------------------------------------------------------------
#define QKN_MAX_HD 512
#define QKN_WARPS 4

// cos and sin of pos * inv_freq[j] for every token of the step, once per step: all layers
// with the same frequencies read the same table.  table[t * half + j] = (cos, sin).
__global__ void rope_table_kernel(const int *__restrict__ tok_pos, const float *__restrict__ inv_freq,
                                  float2 *__restrict__ table, int T_tokens, int half, float mult) {
  pdl_launch();
  pdl_wait();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)T_tokens * half) return;
  const int t = (int)(i / half), j = (int)(i % half);
  float sn, c;
  sincosf((float)tok_pos[t] * inv_freq[j], &sn, &c);
  table[i] = make_float2(c * mult, sn * mult);
}

extern "C" int g2b_rope_table(const int *tok_pos, const float *inv_freq, float *table, int T_tokens,
                              int half, float mult, cudaStream_t stream) {
  if (T_tokens <= 0 || half <= 0) return 0;
  const long long n = (long long)T_tokens * half;
  g2b_launch(rope_table_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, stream, tok_pos, inv_freq,
             (float2 *)table, T_tokens, half, mult);
  return g2b_check_launch("rope_table");
}

// Head sizes 2 * E * LPH (LPH a power of two up to 32, E = 4 or 8) with the rotation over the
// whole head: LPH lanes share a head, so a warp works on 32 / LPH heads of one token at once.
// A lane holds E consecutive elements of the first half and their rotation partners in the
// second half, loaded and stored as vectors; everything stays in registers.  E = 4 gives a
// decode step more lanes per head (shorter chains); E = 8 moves 16 bytes per load for prompts.
#define QKN_FAST_WARPS 8

template <typename T, int LPH, int E>
__global__ void __launch_bounds__(QKN_FAST_WARPS * 32)
qknorm_rope_fast_kernel(
    const T *__restrict__ qkv, int T_tokens, int nh, int nkv,
    const float *__restrict__ q_w, const float *__restrict__ k_w, float eps,
    const float2 *__restrict__ rope,
    const int *__restrict__ tok_pos, const int *__restrict__ tok_seq,
    const int *__restrict__ page_table, int P, T *__restrict__ cache, int page_size,
    T *__restrict__ q_out, T *__restrict__ k_out, T *__restrict__ v_out) {
  pdl_launch();
  pdl_wait();
  constexpr int HPW = 32 / LPH, HD = 2 * E * LPH, HH = E * LPH;
  const unsigned warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const unsigned heads = nh + 2 * nkv;
  const unsigned groups = (heads + HPW - 1) / HPW;
  const unsigned item = blockIdx.x * QKN_FAST_WARPS + warp;
  if (item >= (unsigned)T_tokens * groups) return;
  const unsigned t = item / groups;
  const unsigned h = (item - t * groups) * HPW + lane / LPH;
  const bool valid = h < heads;
  const unsigned hc = valid ? h : heads - 1;
  const int j = E * (lane % LPH);
  const T *src = qkv + ((size_t)t * heads + hc) * HD;
  float a[E], b[E];
  ldE<E>(src + j, a);
  ldE<E>(src + HH + j, b);
  const int kind = hc < (unsigned)nh ? 0 : (hc < (unsigned)(nh + nkv) ? 1 : 2);     // q, k, v
  const float *w = kind == 0 ? q_w : (kind == 1 ? k_w : nullptr);
  T *dst;
  if (kind == 0) {
    dst = q_out + ((size_t)t * nh + hc) * HD;
  } else {
    const unsigned kvh = kind == 1 ? hc - nh : hc - nh - nkv;
    T *flat = kind == 1 ? k_out : v_out;
    if (flat) {
      dst = flat + ((size_t)t * nkv + kvh) * HD;
    } else {
      const int pos = tok_pos[t];
      const int page = page_table[(size_t)tok_seq[t] * P + pos / page_size];
      dst = cache + ((((size_t)page * 2 + (kind - 1)) * nkv + kvh) * page_size + pos % page_size) * HD;
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < E; ++i) {
    ss = fmaf(a[i], a[i], ss);
    ss = fmaf(b[i], b[i], ss);
  }
#pragma unroll
  for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (w) {
    const float inv = 1.f / sqrtf(ss / (float)HD + eps);
    float wa[E], wb[E];
    ldE<E>(w + j, wa);
    ldE<E>(w + HH + j, wb);
#pragma unroll
    for (int i = 0; i < E; ++i) {
      a[i] = (wa[i] * a[i]) * inv;
      b[i] = (wb[i] * b[i]) * inv;
    }
  }
  if (rope && kind != 2) {
    const float2 *cs = rope + (size_t)t * HH + j;
#pragma unroll
    for (int i = 0; i < E; i += 2) {
      const float4 r = *reinterpret_cast<const float4 *>(cs + i);      // (cos, sin) of j+i, j+i+1
      const float a0 = a[i], b0 = b[i], a1 = a[i + 1], b1 = b[i + 1];
      a[i] = a0 * r.x - b0 * r.y;
      b[i] = a0 * r.y + b0 * r.x;
      a[i + 1] = a1 * r.z - b1 * r.w;
      b[i + 1] = a1 * r.w + b1 * r.z;
    }
  }
  if (valid) {
    stE<E>(dst + j, a);
    stE<E>(dst + HH + j, b);
  }
}

// Every other head size and a rotation over part of the head: one warp per (token, head),
// the head staged in shared memory.
template <typename T>
__global__ void __launch_bounds__(QKN_WARPS * 32)
qknorm_rope_cache_kernel(
    const T *__restrict__ qkv, int T_tokens, int nh, int nkv, int hd,
    const float *__restrict__ q_w, const float *__restrict__ k_w, float eps,
    const float2 *__restrict__ rope, int rot_dim,
    const int *__restrict__ tok_pos, const int *__restrict__ tok_seq,
    const int *__restrict__ page_table, int P, T *__restrict__ cache, int page_size,
    T *__restrict__ q_out, T *__restrict__ k_out, T *__restrict__ v_out) {
  pdl_launch();
  pdl_wait();
  __shared__ float buf[QKN_WARPS][QKN_MAX_HD];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int heads = nh + 2 * nkv;
  const long long item = (long long)blockIdx.x * QKN_WARPS + warp;
  if (item >= (long long)T_tokens * heads) return;
  const int t = (int)(item / heads), h = (int)(item % heads);
  const int half = rot_dim >> 1;
  const T *src = qkv + (size_t)t * heads * hd + (size_t)h * hd;
  const int kind = h < nh ? 0 : (h < nh + nkv ? 1 : 2);
  const float *w = kind == 0 ? q_w : (kind == 1 ? k_w : nullptr);
  const float2 *cs = (rope && kind != 2) ? rope + (size_t)t * half : nullptr;
  T *dst;
  if (kind == 0) {
    dst = q_out + (size_t)t * nh * hd + (size_t)h * hd;
  } else {
    const int kvh = kind == 1 ? h - nh : h - nh - nkv;
    T *flat = kind == 1 ? k_out : v_out;
    if (flat) {
      dst = flat + (size_t)t * nkv * hd + (size_t)kvh * hd;
    } else {
      const int pos = tok_pos[t];
      const int page = page_table[(size_t)tok_seq[t] * P + pos / page_size];
      dst = cache + ((((size_t)page * 2 + (kind - 1)) * nkv + kvh) * page_size + pos % page_size) * hd;
    }
  }
  float *x = buf[warp];
  float ss = 0.f;
  for (int j = lane; j < hd; j += 32) {
    const float v = to_f32(src[j]);
    x[j] = v;
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  __syncwarp();
  if (w) {
    const float inv = 1.f / sqrtf(ss / (float)hd + eps);
    for (int j = lane; j < hd; j += 32) x[j] = (w[j] * x[j]) * inv;
    __syncwarp();
  }
  if (cs) {
    for (int j = lane; j < half; j += 32) {
      const float2 r = cs[j];
      const float av = x[j], bv = x[j + half];
      x[j] = av * r.x - bv * r.y;
      x[j + half] = av * r.y + bv * r.x;
    }
    __syncwarp();
  }
  for (int j = lane; j < hd; j += 32) dst[j] = from_f32<T>(x[j]);
}

template <typename T, int LPH, int E>
static void launch_qkn_fast(const void *qkv, int T_tokens, int nh, int nkv, const float *q_w, const float *k_w,
                            float eps, const float *rope_table, const int *tok_pos, const int *tok_seq,
                            const int *page_table, int P, void *cache, int page_size, void *q_out, void *k_out,
                            void *v_out, cudaStream_t stream) {
  const long long items = (long long)T_tokens * ((nh + 2 * nkv + 32 / LPH - 1) / (32 / LPH));
  const unsigned blocks = (unsigned)((items + QKN_FAST_WARPS - 1) / QKN_FAST_WARPS);
  g2b_launch(qknorm_rope_fast_kernel<T, LPH, E>, dim3(blocks), dim3(QKN_FAST_WARPS * 32), 0, stream,
             (const T *)qkv, T_tokens, nh, nkv, q_w, k_w, eps, (const float2 *)rope_table, tok_pos, tok_seq,
             page_table, P, (T *)cache, page_size, (T *)q_out, (T *)k_out, (T *)v_out);
}

extern "C" int g2b_qknorm_rope_cache(const void *qkv, int dtype, int T_tokens, int nh, int nkv,
                                     int hd, const float *q_w, const float *k_w, float eps,
                                     const float *rope_table, int rot_dim, const int *tok_pos,
                                     const int *tok_seq, const int *page_table, int P,
                                     void *cache, int page_size, void *q_out, void *k_out,
                                     void *v_out, cudaStream_t stream) {
  if (T_tokens <= 0) return 0;
  if (dtype != G2B_F32 && dtype != G2B_BF16) G2B_REFUSE("qknorm_rope_cache: unknown dtype %d", dtype);
  if (hd <= 0 || hd > QKN_MAX_HD)
    G2B_REFUSE("qknorm_rope_cache: head_dim %d outside 1..%d", hd, QKN_MAX_HD);
  if (rope_table && (rot_dim <= 0 || rot_dim > hd || (rot_dim & 1)))
    G2B_REFUSE("qknorm_rope_cache: rotary_dim %d must be even and at most head_dim %d", rot_dim, hd);
  if ((k_out == nullptr) != (v_out == nullptr))
    G2B_REFUSE("qknorm_rope_cache: k_out and v_out must be given together");
  if (nkv > 0 && !k_out && (!cache || !page_table || page_size <= 0))
    G2B_REFUSE("qknorm_rope_cache: no cache to write to");
  const int heads = nh + 2 * nkv;
  // eight elements per lane and half for prompts (many rows), four for the few rows of a decode step
  const bool wide = hd % 16 == 0 && hd >= 32 && (long long)T_tokens * heads >= 4096;
  const int epl = wide ? 8 : 4;
  const int lph = hd / (2 * epl);
  const bool aligned = (((uintptr_t)qkv | (uintptr_t)q_out | (uintptr_t)cache | (uintptr_t)k_out |
                         (uintptr_t)v_out | (uintptr_t)rope_table | (uintptr_t)q_w | (uintptr_t)k_w) & 15) == 0;
  const bool fast = aligned && hd % (2 * epl) == 0 && lph >= 2 && lph <= 32 && (lph & (lph - 1)) == 0 &&
                    (!rope_table || rot_dim == hd) && (long long)T_tokens * heads < (1ll << 31);
  if (fast) {
#define G2B_QKN_FAST(L)                                                                                     \
  case L:                                                                                                   \
    if (dtype == G2B_F32 && wide)                                                                           \
      launch_qkn_fast<float, L, 8>(qkv, T_tokens, nh, nkv, q_w, k_w, eps, rope_table, tok_pos, tok_seq,     \
                                   page_table, P, cache, page_size, q_out, k_out, v_out, stream);           \
    else if (dtype == G2B_F32)                                                                              \
      launch_qkn_fast<float, L, 4>(qkv, T_tokens, nh, nkv, q_w, k_w, eps, rope_table, tok_pos, tok_seq,     \
                                   page_table, P, cache, page_size, q_out, k_out, v_out, stream);           \
    else if (wide)                                                                                          \
      launch_qkn_fast<bf16, L, 8>(qkv, T_tokens, nh, nkv, q_w, k_w, eps, rope_table, tok_pos, tok_seq,      \
                                  page_table, P, cache, page_size, q_out, k_out, v_out, stream);            \
    else                                                                                                    \
      launch_qkn_fast<bf16, L, 4>(qkv, T_tokens, nh, nkv, q_w, k_w, eps, rope_table, tok_pos, tok_seq,      \
                                  page_table, P, cache, page_size, q_out, k_out, v_out, stream);            \
    break;
    switch (lph) {
      G2B_QKN_FAST(2) G2B_QKN_FAST(4) G2B_QKN_FAST(8) G2B_QKN_FAST(16) G2B_QKN_FAST(32)
    }
#undef G2B_QKN_FAST
    return g2b_check_launch("qknorm_rope_cache");
  }
  const long long items = (long long)T_tokens * heads;
  const unsigned blocks = (unsigned)((items + QKN_WARPS - 1) / QKN_WARPS);
  if (dtype == G2B_F32)
    g2b_launch(qknorm_rope_cache_kernel<float>, dim3(blocks), dim3(QKN_WARPS * 32), 0, stream,
        (const float *)qkv, T_tokens, nh, nkv, hd, q_w, k_w, eps, (const float2 *)rope_table, rot_dim,
        tok_pos, tok_seq, page_table, P, (float *)cache, page_size, (float *)q_out, (float *)k_out,
        (float *)v_out);
  else
    g2b_launch(qknorm_rope_cache_kernel<bf16>, dim3(blocks), dim3(QKN_WARPS * 32), 0, stream,
        (const bf16 *)qkv, T_tokens, nh, nkv, hd, q_w, k_w, eps, (const float2 *)rope_table, rot_dim,
        tok_pos, tok_seq, page_table, P, (bf16 *)cache, page_size, (bf16 *)q_out, (bf16 *)k_out,
        (bf16 *)v_out);
  return g2b_check_launch("qknorm_rope_cache");
}

// ---------------------------------------------------------------------------
// cache write alone: k, v [T, nkv*hd] -> the layer's pages
// ---------------------------------------------------------------------------
template <typename T>
__global__ void cache_write_kernel(const T *__restrict__ k, const T *__restrict__ v, int nkv,
                                   int hd, const int *__restrict__ tok_pos,
                                   const int *__restrict__ tok_seq,
                                   const int *__restrict__ page_table, int P,
                                   T *__restrict__ cache, int page_size) {
  pdl_launch();
  pdl_wait();
  const int t = blockIdx.x;
  const int pos = tok_pos[t];
  const int page = page_table[(size_t)tok_seq[t] * P + pos / page_size];
  const int n = nkv * hd;
  for (int i = threadIdx.x; i < 2 * n; i += blockDim.x) {
    const int which = i / n, r = i % n, kvh = r / hd, j = r % hd;
    const T val = (which == 0 ? k : v)[(size_t)t * n + r];
    cache[((((size_t)page * 2 + which) * nkv + kvh) * page_size + pos % page_size) * hd + j] = val;
  }
}

extern "C" int g2b_cache_write(const void *k, const void *v, int dtype, int T_tokens, int nkv,
                               int hd, const int *tok_pos, const int *tok_seq,
                               const int *page_table, int P, void *cache, int page_size,
                               cudaStream_t stream) {
  if (T_tokens <= 0) return 0;
  if (dtype == G2B_F32)
    g2b_launch(cache_write_kernel<float>, dim3(T_tokens), dim3(128), 0, stream, 
        (const float *)k, (const float *)v, nkv, hd, tok_pos, tok_seq, page_table, P,
        (float *)cache, page_size);
  else if (dtype == G2B_BF16)
    g2b_launch(cache_write_kernel<bf16>, dim3(T_tokens), dim3(128), 0, stream, 
        (const bf16 *)k, (const bf16 *)v, nkv, hd, tok_pos, tok_seq, page_table, P, (bf16 *)cache,
        page_size);
  else
    G2B_REFUSE("cache_write: unknown dtype %d", dtype);
  return g2b_check_launch("cache_write");
}

// ---------------------------------------------------------------------------
// RMS norm with a token shift: h = w * x / rms(x) for the readers that take the token as it is,
// and hs = h + (h_prev - h) * mu for the reader that looks one token back.  h_prev is the normed
// row of the token before in the sequence: the row above in this step, or the sequence's kept row
// (`state` [slots, H] float; zeros in front of position 0).  The block of a sequence's first row of
// the step reads the kept row and then replaces it with the normed LAST row of the step, so nobody
// else touches that slot's place in this launch.  One block per token.
//   seq_meta [B,4]: first row of the step, rows, tokens before the step, slot; null: one token per
//   sequence, its position in tok_pos and its slot in seq_slots.
// ---------------------------------------------------------------------------
template <typename TO>
__global__ void __launch_bounds__(256)
norm_shift_kernel(const float *__restrict__ x, const float *__restrict__ w, const float *__restrict__ mu,
                  float *__restrict__ state, const int *__restrict__ tok_seq, const int *__restrict__ tok_pos,
                  const int *__restrict__ seq_slots, const int *__restrict__ seq_meta,
                  TO *__restrict__ h_out, TO *__restrict__ hs_out, int H, float eps) {
  pdl_launch();
  pdl_wait();
  __shared__ float scratch[32];
  const int t = blockIdx.x;
  const int b = tok_seq[t];
  // without the table of sequences the step is one token per sequence
  const int first_row = seq_meta ? seq_meta[4 * b + 0] : t, n = seq_meta ? seq_meta[4 * b + 1] : 1;
  const int past = seq_meta ? seq_meta[4 * b + 2] : tok_pos[t];
  const int slot = seq_meta ? seq_meta[4 * b + 3] : seq_slots[b];
  const bool first = t == first_row;
  const float *xr = x + (size_t)t * H;
  float ss = 0.f;
  for (int j = threadIdx.x; j < H; j += blockDim.x) ss = fmaf(xr[j], xr[j], ss);
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)H + eps);
  float inv_prev = 0.f;
  const float *xp = xr - H;                          // the row above, where it is the same sequence's
  if (!first) {
    float sp = 0.f;
    for (int j = threadIdx.x; j < H; j += blockDim.x) sp = fmaf(xp[j], xp[j], sp);
    inv_prev = 1.f / sqrtf(block_sum(sp, scratch) / (float)H + eps);
  }
  float *kept = state + (size_t)slot * H;
  const bool from_state = first && past > 0;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    const float g = w ? w[j] : 1.f;
    const float h = (g * xr[j]) * inv;
    const float hp = first ? (from_state ? kept[j] : 0.f) : (g * xp[j]) * inv_prev;
    h_out[(size_t)t * H + j] = from_f32<TO>(h);
    hs_out[(size_t)t * H + j] = from_f32<TO>(fmaf(hp - h, mu[j], h));
  }
  if (!first) return;
  // this block alone reads and writes the slot's kept row; every read above is over
  const float *xl = x + (size_t)(first_row + n - 1) * H;
  float inv_last = inv;
  if (n > 1) {
    float sl = 0.f;
    for (int j = threadIdx.x; j < H; j += blockDim.x) sl = fmaf(xl[j], xl[j], sl);
    inv_last = 1.f / sqrtf(block_sum(sl, scratch) / (float)H + eps);
  }
  __syncthreads();
  for (int j = threadIdx.x; j < H; j += blockDim.x) kept[j] = ((w ? w[j] : 1.f) * xl[j]) * inv_last;
}

extern "C" int g2b_norm_shift(const float *x, const float *w, const float *mu, float *state, const int *tok_seq,
                              const int *tok_pos, const int *seq_slots, const int *seq_meta, int T_tokens, int H,
                              float eps, void *h_out, void *hs_out, int out_dtype, cudaStream_t stream) {
  if (T_tokens <= 0) return 0;
  if (!mu || !state || !tok_seq || (!seq_meta && (!tok_pos || !seq_slots)))
    G2B_REFUSE("norm_shift: shift weights, kept rows and the step's tables are needed");
  if (out_dtype == G2B_F32)
    g2b_launch(norm_shift_kernel<float>, dim3(T_tokens), dim3(256), 0, stream, x, w, mu, state, tok_seq, tok_pos, seq_slots, seq_meta,
               (float *)h_out, (float *)hs_out, H, eps);
  else if (out_dtype == G2B_BF16)
    g2b_launch(norm_shift_kernel<bf16>, dim3(T_tokens), dim3(256), 0, stream, x, w, mu, state, tok_seq, tok_pos, seq_slots, seq_meta,
               (bf16 *)h_out, (bf16 *)hs_out, H, eps);
  else
    G2B_REFUSE("norm_shift: unknown output dtype %d", out_dtype);
  return g2b_check_launch("norm_shift");
}

// ---------------------------------------------------------------------------
// One row mixed with the row in front of it in several ways: out[i, t] = h_t + (h_prev - h_t) * mu[i], i < n, 32-bit
// arithmetic on rows of the compute type.  h_prev is the row above in this step where it is the same sequence's, else
// the sequence's kept row (`kept` [slots, H] in the compute type; zeros in front of position 0).  The block of a
// sequence's first row reads the kept row and then replaces it with the sequence's last row of the step (an input), so
// nobody else touches that slot's place in this launch.  A block per (token, stretch of columns); tables as above.
// ---------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
shift_mix_kernel(const T *__restrict__ h, int h_stride, const float *__restrict__ mu, int n, T *__restrict__ kept,
                 const int *__restrict__ tok_seq, const int *__restrict__ tok_pos, const int *__restrict__ seq_slots,
                 const int *__restrict__ seq_meta, int n_tokens, int H, T *__restrict__ out) {
  pdl_launch();
  pdl_wait();
  const int t = blockIdx.x, j = blockIdx.y * 256 + threadIdx.x;
  if (j >= H) return;
  const int b = tok_seq[t];
  const int first_row = seq_meta ? seq_meta[4 * b + 0] : t, rows = seq_meta ? seq_meta[4 * b + 1] : 1;
  const int past = seq_meta ? seq_meta[4 * b + 2] : tok_pos[t];
  const int slot = seq_meta ? seq_meta[4 * b + 3] : seq_slots[b];
  const bool first = t == first_row;
  T *keep = kept + (size_t)slot * H + j;
  const T *own = h + (size_t)t * h_stride + j;
  const float x = to_f32(*own);
  const float d = (first ? (past > 0 ? to_f32(*keep) : 0.f) : to_f32(*(own - h_stride))) - x;
  for (int m = 0; m < n; ++m) out[((size_t)m * n_tokens + t) * H + j] = from_f32<T>(fmaf(d, mu[(size_t)m * H + j], x));
  if (first) *keep = h[(size_t)(first_row + rows - 1) * h_stride + j];       // this thread alone reads and writes that entry
}

// N (4 or 8) bfloat16 neighbours a thread
template <int N>
__global__ void __launch_bounds__(256)
shift_mix_vec_kernel(const bf16 *__restrict__ h, int h_stride, const float *__restrict__ mu, int n, bf16 *__restrict__ kept,
                  const int *__restrict__ tok_seq, const int *__restrict__ tok_pos, const int *__restrict__ seq_slots,
                  const int *__restrict__ seq_meta, int n_tokens, int H, bf16 *__restrict__ out) {
  pdl_launch();
  pdl_wait();
  const int t = blockIdx.x, j = (blockIdx.y * blockDim.x + threadIdx.x) * N;
  if (j >= H) return;
  const int b = tok_seq[t];
  const int first_row = seq_meta ? seq_meta[4 * b + 0] : t, rows = seq_meta ? seq_meta[4 * b + 1] : 1;
  const int past = seq_meta ? seq_meta[4 * b + 2] : tok_pos[t];
  const int slot = seq_meta ? seq_meta[4 * b + 3] : seq_slots[b];
  const bool first = t == first_row;
  bf16 *keep = kept + (size_t)slot * H + j;
  const bf16 *own = h + (size_t)t * h_stride + j;
  float x[N], d[N];
  ldE<N>(own, x);
  if (!first) {
    ldE<N>(own - h_stride, d);
  } else if (past > 0) {
    ldE<N>(keep, d);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) d[i] = 0.f;
  }
#pragma unroll
  for (int i = 0; i < N; ++i) d[i] -= x[i];
  for (int m = 0; m < n; ++m) {
    float r[N];
#pragma unroll
    for (int i = 0; i < N; i += 4) {
      const float4 w = *reinterpret_cast<const float4 *>(mu + (size_t)m * H + j + i);
      r[i] = fmaf(d[i], w.x, x[i]), r[i + 1] = fmaf(d[i + 1], w.y, x[i + 1]);
      r[i + 2] = fmaf(d[i + 2], w.z, x[i + 2]), r[i + 3] = fmaf(d[i + 3], w.w, x[i + 3]);
    }
    stE<N>(out + ((size_t)m * n_tokens + t) * H + j, r);
  }
  if (first) {                                       // this thread alone reads and writes these entries of the slot
    ldE<N>(h + (size_t)(first_row + rows - 1) * h_stride + j, x);
    stE<N>(keep, x);
  }
}

extern "C" int g2b_shift_mix(const void *h, int h_stride, const float *mu, int n, void *kept, const int *tok_seq,
                             const int *tok_pos, const int *seq_slots, const int *seq_meta, int T_tokens, int H, void *out,
                             int dtype, cudaStream_t stream) {
  if (T_tokens <= 0) return 0;
  if (!mu || n <= 0 || !kept || !tok_seq || (!seq_meta && (!tok_pos || !seq_slots)))
    G2B_REFUSE("shift_mix: mixing weights, kept rows and the step's tables are needed");
  const uintptr_t at = (uintptr_t)h | (uintptr_t)kept | (uintptr_t)out;
  if (dtype == G2B_BF16 && H % 4 == 0 && h_stride % 4 == 0 && !(at & 7) && !((uintptr_t)mu & 15)) {
    const bool wide = H % 8 == 0 && h_stride % 8 == 0 && !(at & 15) && T_tokens >= 64;
    const int pieces = H / (wide ? 8 : 4), threads = pieces >= 256 ? 256 : (pieces + 31) / 32 * 32;
    const dim3 grid(T_tokens, (pieces + threads - 1) / threads);
    if (grid.y > 65535) G2B_REFUSE("shift_mix: rows of %d", H);
    g2b_launch(wide ? shift_mix_vec_kernel<8> : shift_mix_vec_kernel<4>, grid, dim3(threads), 0, stream, (const bf16 *)h, h_stride, mu,
               n, (bf16 *)kept, tok_seq, tok_pos, seq_slots, seq_meta, T_tokens, H, (bf16 *)out);
    return g2b_check_launch("shift_mix");
  }
  const dim3 grid(T_tokens, (H + 255) / 256);
  if (grid.y > 65535) G2B_REFUSE("shift_mix: rows of %d", H);
  if (dtype == G2B_F32)
    g2b_launch(shift_mix_kernel<float>, grid, dim3(256), 0, stream, (const float *)h, h_stride, mu, n, (float *)kept, tok_seq,
               tok_pos, seq_slots, seq_meta, T_tokens, H, (float *)out);
  else if (dtype == G2B_BF16)
    g2b_launch(shift_mix_kernel<bf16>, grid, dim3(256), 0, stream, (const bf16 *)h, h_stride, mu, n, (bf16 *)kept, tok_seq,
               tok_pos, seq_slots, seq_meta, T_tokens, H, (bf16 *)out);
  else
    G2B_REFUSE("shift_mix: unknown dtype %d", dtype);
  return g2b_check_launch("shift_mix");
}

// ---------------------------------------------------------------------------
// SiLU gate on a fused gate/up projection.  Rows of the fused matrix alternate in
// blocks of `blk`: columns [2*blk*b, 2*blk*b+blk) are gate_{blk*b ..}, the next blk are
// up_{blk*b ..}; blk == I means "all gates, then all ups".
//   out[t, i] = (g / (1 + exp(-g))) * u, or another gate of the form in glu.cuh
// ---------------------------------------------------------------------------
template <typename T>
__global__ void swiglu_kernel(const T *__restrict__ gu, T *__restrict__ out, long long total,
                              int I, int blk, GluForm glu) {
  pdl_launch();
  pdl_wait();
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= total) return;
  const long long t = idx / I;
  const int i = (int)(idx % I);
  const int b = i / blk, r = i % blk;
  const T *row = gu + (size_t)t * 2 * I;
  const float g = to_f32(row[(size_t)2 * blk * b + r]);
  const float u = to_f32(row[(size_t)2 * blk * b + blk + r]);
  out[idx] = from_f32<T>(glu_value(g, u, glu));
}

// The same in bfloat16 for blocks of a multiple of eight: a thread takes eight neighbouring outputs,
// their gates and their ups as one 16-byte load each.
__global__ void __launch_bounds__(256)
swiglu8_kernel(const bf16 *__restrict__ gu, bf16 *__restrict__ out, long long total8, int I, int blk, GluForm glu) {
  pdl_launch();
  pdl_wait();
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= total8) return;
  const int per_row = I / 8;
  const long long t = idx / per_row;
  const int i = (int)(idx % per_row) * 8;
  const int b = i / blk, r = i % blk;
  const bf16 *src = gu + (size_t)t * 2 * I + (size_t)2 * blk * b + r;
  const uint4 gv = __ldg(reinterpret_cast<const uint4 *>(src));
  const uint4 uv = __ldg(reinterpret_cast<const uint4 *>(src + blk));
  const unsigned int gw[4] = {gv.x, gv.y, gv.z, gv.w}, uw[4] = {uv.x, uv.y, uv.z, uv.w};
  unsigned int ow[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&gw[e]));
    const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&uw[e]));
    const __nv_bfloat162 ob = __floats2bfloat162_rn(glu_value(g.x, u.x, glu), glu_value(g.y, u.y, glu));
    ow[e] = *reinterpret_cast<const unsigned int *>(&ob);
  }
  *reinterpret_cast<uint4 *>(out + (size_t)t * I + i) = make_uint4(ow[0], ow[1], ow[2], ow[3]);
}

extern "C" int g2b_swiglu(const void *gu, int dtype, int T_tokens, int I, int blk, void *out,
                          float glu_limit, float glu_offset, float glu_c1, float glu_c3, cudaStream_t stream) {
  const GluForm glu = {glu_limit, glu_offset, glu_c1, glu_c3};
  if (T_tokens <= 0) return 0;
  if (I <= 0 || blk <= 0 || I % blk) G2B_REFUSE("swiglu: block %d does not divide width %d", blk, I);
  const long long total = (long long)T_tokens * I;
  if (dtype == G2B_BF16 && blk % 8 == 0 && !(((uintptr_t)gu | (uintptr_t)out) & 15)) {
    const long long total8 = total / 8;
    g2b_launch(swiglu8_kernel, dim3((unsigned)((total8 + 255) / 256)), dim3(256), 0, stream, (const bf16 *)gu, (bf16 *)out,
               total8, I, blk, glu);
    return g2b_check_launch("swiglu");
  }
  const unsigned blocks = (unsigned)((total + 255) / 256);
  if (dtype == G2B_F32)
    g2b_launch(swiglu_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float *)gu, (float *)out, total, I, blk, glu);
  else if (dtype == G2B_BF16)
    g2b_launch(swiglu_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, (const bf16 *)gu, (bf16 *)out, total, I, blk, glu);
  else
    G2B_REFUSE("swiglu: unknown dtype %d", dtype);
  return g2b_check_launch("swiglu");
}

// ---------------------------------------------------------------------------
// decode bookkeeping on the device, for steps replayed from a CUDA graph:
// positions advance by one.
// ---------------------------------------------------------------------------
__global__ void advance_positions_kernel(int *tok_pos, int n) {
  pdl_launch();
  pdl_wait();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) tok_pos[i] += 1;
}

extern "C" int g2b_advance_positions(int *tok_pos, int n, cudaStream_t stream) {
  if (n <= 0) return 0;
  g2b_launch(advance_positions_kernel, dim3((n + 127) / 128), dim3(128), 0, stream, tok_pos, n);
  return g2b_check_launch("advance_positions");
}

// Undoes the bookkeeping of one decode step that was launched ahead and is not wanted after
// all: positions go back by one and, when that step drew a random number, so do the draw
// counters of the sequences' sampling records, and the count of its recent ids when that step added one.
// (words 3 and 4 of a record: the draw counter and the count of ids in the ring of recent ids;
// the id that the step wrote stays in the ring, one place past the window)
__global__ void rewind_step_kernel(int *tok_pos, int n, int *seq_state, int words, const int *slots, int undo_draw,
                                   int undo_recent) {
  pdl_launch();
  pdl_wait();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  tok_pos[i] = max(tok_pos[i] - 1, 0);          // a row of padding may have been set back to 0 since the step
  if (undo_draw) seq_state[(size_t)slots[i] * words + 3] -= 1;
  if (undo_recent) seq_state[(size_t)slots[i] * words + 4] -= 1;
}

extern "C" int g2b_rewind_step(int *tok_pos, int n, int *seq_state, int words, const int *slots, int undo_draw,
                               int undo_recent, cudaStream_t stream) {
  if (n <= 0) return 0;
  if ((undo_draw || undo_recent) && (!seq_state || !slots || words < 5))
    G2B_REFUSE("rewind_step: no sampling records to rewind");
  g2b_launch(rewind_step_kernel, dim3((n + 127) / 128), dim3(128), 0, stream, tok_pos, n, seq_state, words, slots,
             undo_draw, undo_recent);
  return g2b_check_launch("rewind_step");
}

// ---------------------------------------------------------------------------
// a norm without statistics, sublayer results joined with a weight per channel,
// and the squared rectifier
// ---------------------------------------------------------------------------
// out[r] = tanh(alpha x[row_r]) * w + b: nothing is summed over the row, so a thread takes four
// neighbours of any row; alpha is one number, read from the device.
template <typename TO>
__global__ void __launch_bounds__(256)
tanh_norm_kernel(const float *__restrict__ x, const float *__restrict__ alpha, const float *__restrict__ w,
                 const float *__restrict__ b, const int *__restrict__ rows, TO *__restrict__ out, int n_rows, int H) {
  pdl_launch();
  pdl_wait();
  const float a = alpha[0];
  const long long total = (long long)n_rows * H;
  if ((H & 3) == 0) {
    const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) * 4;
    if (i >= total) return;
    const int r = (int)(i / H), k = (int)(i % H);
    const float4 v = *reinterpret_cast<const float4 *>(x + (size_t)(rows ? rows[r] : r) * H + k);
    const float4 g = *reinterpret_cast<const float4 *>(w + k), c = *reinterpret_cast<const float4 *>(b + k);
    store4(out + i, fmaf(tanhf(a * v.x), g.x, c.x), fmaf(tanhf(a * v.y), g.y, c.y), fmaf(tanhf(a * v.z), g.z, c.z),
           fmaf(tanhf(a * v.w), g.w, c.w));
    return;
  }
  for (int j = 0; j < 4; ++j) {
    const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) * 4 + j;
    if (i >= total) return;
    const int r = (int)(i / H), k = (int)(i % H);
    out[i] = from_f32<TO>(fmaf(tanhf(a * x[(size_t)(rows ? rows[r] : r) * H + k]), w[k], b[k]));
  }
}

extern "C" int g2b_tanh_norm(const float *x, const float *alpha, const float *w, const float *b, const int *rows,
                             int n_rows, int H, void *out, int out_dtype, cudaStream_t stream) {
  if (n_rows <= 0 || H <= 0) return 0;
  const long long quads = ((long long)n_rows * H + 3) / 4;
  const unsigned blocks = (unsigned)((quads + 255) / 256);
  if (out_dtype == G2B_F32)
    g2b_launch(tanh_norm_kernel<float>, dim3(blocks), dim3(256), 0, stream, x, alpha, w, b, rows, (float *)out, n_rows, H);
  else if (out_dtype == G2B_BF16)
    g2b_launch(tanh_norm_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, x, alpha, w, b, rows, (bf16 *)out, n_rows, H);
  else
    G2B_REFUSE("tanh_norm: unknown dtype %d", out_dtype);
  return g2b_check_launch("tanh_norm");
}

// x += y1 * s1 + y2 * s2 (s: one number per channel; y2 may be absent), all float.  With `alpha`: the new rows
// once more as tanh(alpha x) * w + b in the compute type, which is what the next layer's norm would compute.
template <typename TO>
__global__ void __launch_bounds__(256)
scaled_join_kernel(float *__restrict__ x, const float *__restrict__ y1, const float *__restrict__ s1,
                   const float *__restrict__ y2, const float *__restrict__ s2, long long total, int H,
                   const float *__restrict__ alpha, const float *__restrict__ nw, const float *__restrict__ nb,
                   TO *__restrict__ normed) {
  pdl_launch();
  pdl_wait();
  if ((H & 3) == 0) {
    const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) * 4;
    if (i >= total) return;
    const int k = (int)(i % H);
    float4 v = *reinterpret_cast<float4 *>(x + i);
    const float4 a = *reinterpret_cast<const float4 *>(y1 + i), ga = *reinterpret_cast<const float4 *>(s1 + k);
    float4 add = make_float4(a.x * ga.x, a.y * ga.y, a.z * ga.z, a.w * ga.w);
    if (y2) {
      const float4 c = *reinterpret_cast<const float4 *>(y2 + i), gc = *reinterpret_cast<const float4 *>(s2 + k);
      add.x = fmaf(c.x, gc.x, add.x); add.y = fmaf(c.y, gc.y, add.y);
      add.z = fmaf(c.z, gc.z, add.z); add.w = fmaf(c.w, gc.w, add.w);
    }
    v.x += add.x; v.y += add.y; v.z += add.z; v.w += add.w;
    *reinterpret_cast<float4 *>(x + i) = v;
    if (alpha) {
      const float a = alpha[0];
      const float4 g = *reinterpret_cast<const float4 *>(nw + k), c = *reinterpret_cast<const float4 *>(nb + k);
      store4(normed + i, fmaf(tanhf(a * v.x), g.x, c.x), fmaf(tanhf(a * v.y), g.y, c.y), fmaf(tanhf(a * v.z), g.z, c.z),
             fmaf(tanhf(a * v.w), g.w, c.w));
    }
    return;
  }
  for (int j = 0; j < 4; ++j) {
    const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) * 4 + j;
    if (i >= total) return;
    const int k = (int)(i % H);
    float add = y1[i] * s1[k];
    if (y2) add = fmaf(y2[i], s2[k], add);
    const float v = x[i] + add;
    x[i] = v;
    if (alpha) normed[i] = from_f32<TO>(fmaf(tanhf(alpha[0] * v), nw[k], nb[k]));
  }
}

extern "C" int g2b_scaled_join(float *x, const float *y1, const float *s1, const float *y2, const float *s2,
                               int n_rows, int H, const float *alpha, const float *nw, const float *nb, void *normed,
                               int normed_dtype, cudaStream_t stream) {
  if (n_rows <= 0 || H <= 0) return 0;
  const long long total = (long long)n_rows * H, quads = (total + 3) / 4;
  const dim3 grid((unsigned)((quads + 255) / 256));
  if (!alpha || normed_dtype == G2B_F32)
    g2b_launch(scaled_join_kernel<float>, grid, dim3(256), 0, stream, x, y1, s1, y2, s2, total, H, alpha, nw, nb,
               (float *)normed);
  else if (normed_dtype == G2B_BF16)
    g2b_launch(scaled_join_kernel<bf16>, grid, dim3(256), 0, stream, x, y1, s1, y2, s2, total, H, alpha, nw, nb,
               (bf16 *)normed);
  else
    G2B_REFUSE("scaled_join: unknown dtype %d", normed_dtype);
  return g2b_check_launch("scaled_join");
}

// out = max(z, 0)^2; z rows may lie apart (columns of a wider product's output)
template <typename T>
__global__ void __launch_bounds__(256)
relu2_kernel(const T *__restrict__ z, int z_stride, T *__restrict__ out, long long total, int F) {
  pdl_launch();
  pdl_wait();
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= total) return;
  const float v = fmaxf(to_f32(z[(size_t)(i / F) * z_stride + (i % F)]), 0.f);
  out[i] = from_f32<T>(v * v);
}

__global__ void __launch_bounds__(256)
relu2x8_kernel(const bf16 *__restrict__ z, int z_stride, bf16 *__restrict__ out, long long total8, int F) {
  pdl_launch();
  pdl_wait();
  const long long i8 = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i8 >= total8) return;
  const long long i = i8 * 8;
  const uint4 raw = *reinterpret_cast<const uint4 *>(z + (size_t)(i / F) * z_stride + (i % F));
  const __nv_bfloat162 *in = reinterpret_cast<const __nv_bfloat162 *>(&raw);
  uint4 o;
  __nv_bfloat162 *op = reinterpret_cast<__nv_bfloat162 *>(&o);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    float2 f = __bfloat1622float2(in[j]);
    f.x = fmaxf(f.x, 0.f); f.y = fmaxf(f.y, 0.f);
    op[j] = __floats2bfloat162_rn(f.x * f.x, f.y * f.y);
  }
  *reinterpret_cast<uint4 *>(out + i) = o;
}

extern "C" int g2b_relu2(const void *z, int z_stride, int dtype, int T_tokens, int F, void *out, cudaStream_t stream) {
  if (T_tokens <= 0 || F <= 0) return 0;
  const long long total = (long long)T_tokens * F;
  if (dtype == G2B_BF16 && F % 8 == 0 && z_stride % 8 == 0 && !(((uintptr_t)z | (uintptr_t)out) & 15)) {
    g2b_launch(relu2x8_kernel, dim3((unsigned)((total / 8 + 255) / 256)), dim3(256), 0, stream, (const bf16 *)z, z_stride,
               (bf16 *)out, total / 8, F);
    return g2b_check_launch("relu2");
  }
  const unsigned blocks = (unsigned)((total + 255) / 256);
  if (dtype == G2B_F32)
    g2b_launch(relu2_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float *)z, z_stride, (float *)out, total, F);
  else if (dtype == G2B_BF16)
    g2b_launch(relu2_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, (const bf16 *)z, z_stride, (bf16 *)out, total, F);
  else
    G2B_REFUSE("relu2: unknown dtype %d", dtype);
  return g2b_check_launch("relu2");
}

// out = z * sigmoid(z (c1 + c3 z^2)): an activation of glu.cuh's form without a second input
template <typename T>
__global__ void __launch_bounds__(256)
act_form_kernel(const T *__restrict__ z, int z_stride, T *__restrict__ out, long long total, int F, GluForm form) {
  pdl_launch();
  pdl_wait();
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= total) return;
  out[i] = from_f32<T>(act_value(to_f32(z[(size_t)(i / F) * z_stride + (i % F)]), form));
}

extern "C" int g2b_act_form(const void *z, int z_stride, int dtype, int T_tokens, int F, void *out, float c1, float c3,
                            cudaStream_t stream) {
  if (T_tokens <= 0 || F <= 0) return 0;
  const long long total = (long long)T_tokens * F;
  const unsigned blocks = (unsigned)((total + 255) / 256);
  const GluForm form = {INFINITY, 0.f, c1, c3};
  if (dtype == G2B_F32)
    g2b_launch(act_form_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float *)z, z_stride, (float *)out, total, F, form);
  else if (dtype == G2B_BF16)
    g2b_launch(act_form_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, (const bf16 *)z, z_stride, (bf16 *)out, total, F, form);
  else
    G2B_REFUSE("act_form: unknown dtype %d", dtype);
  return g2b_check_launch("act_form");
}
