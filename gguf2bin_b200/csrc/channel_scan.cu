// A matrix state per head with a decay per KEY CHANNEL (gated linear attention, time mixing with a bonus):
//   S <- diag(a_t) S + k_t v_t^T,   o_t = S^T q_t,   S [D, V] per head
// with z_t = W_low l_t + bias: one number per token, head and key channel, from a vector l_t of R entries per token
// (R small; its entries may pass tanh first), and a_t = sigmoid(z_t)^(1/tau) or exp(-exp(z_t)).
// With a bonus u [H, D] the read-out comes before the update and the token's own key counts u times:
//   o_t = (S + diag(u) k_t v_t^T)^T q_t = S^T q_t + (sum_d q_d u_d k_d) v_t,   then the update.
// Everything but the inputs q, k, v, l, W_low is 32-bit (l may be, too).
// The state is stored column by column ([slot, head, V, D]), as in seq_mix.cu.
//
//   channel_step      one token per sequence: decays, update and read-out in one launch
//   channel_prep      prompts: decays, scaled queries and keys as float rows, once for all columns
//   channel_segment   a block walks one segment of a sequence (a tile of the step's work list) for a range of a
//                     head's columns.  First launch, only where a sequence has several segments: every segment
//                     but the last from a zero state, which leaves its end state and the product of its decays.
//   channel_carry     the states in front of the segments, one after the other: S' = P S + E (the recurrence is
//                     linear in S, and P <= 1: nothing is divided)
//   channel_segment   second launch: every segment from the state in front of it, with read-outs
//
// What a token gets depends on the tokens before it in its sequence only; where segments begin changes the
// order of a few additions.
#include "common.cuh"

G2B_DEFINE_LAST_ERROR

#define CS_MAX_D 512
#define CS_MAX_R 1024

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// sigmoid(z)^(1/tau) through its logarithm
__device__ __forceinline__ float decay_of(float z, float inv_tau) { return expf(-softplus_f(-z) * inv_tau); }
enum { DECAY_SIGMOID_ROOT = 0, DECAY_DOUBLE_EXP = 1 };

// sum over r of w[r] * low[r], R a multiple of eight, ascending r; low on 16 bytes
__device__ __forceinline__ float low_dot(const float *w, const float *low, int R, float acc) {
  for (int r = 0; r < R; r += 4) {
    const float4 a = __ldg(reinterpret_cast<const float4 *>(w + r)), l = *reinterpret_cast<const float4 *>(low + r);
    acc = fmaf(a.x, l.x, acc), acc = fmaf(a.y, l.y, acc);
    acc = fmaf(a.z, l.z, acc), acc = fmaf(a.w, l.w, acc);
  }
  return acc;
}
__device__ __forceinline__ float low_dot(const bf16 *w, const float *low, int R, float acc) {
  for (int r = 0; r < R; r += 8) {
    const uint4 a = __ldg(reinterpret_cast<const uint4 *>(w + r));
    const unsigned int u[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
    for (int i = 0; i < 4; i += 2) {
      const float4 l = *reinterpret_cast<const float4 *>(low + r + 2 * i);
      acc = fmaf(__uint_as_float(u[i] << 16), l.x, acc);
      acc = fmaf(__uint_as_float(u[i] & 0xffff0000u), l.y, acc);
      acc = fmaf(__uint_as_float(u[i + 1] << 16), l.z, acc);
      acc = fmaf(__uint_as_float(u[i + 1] & 0xffff0000u), l.w, acc);
    }
  }
  return acc;
}

struct ChannelIn {
  const void *q, *k, *v, *low;        // compute type; rows of wider buffers
  int q_stride, k_stride, v_stride, low_stride;
  const void *w_low;                  // [H * D, R] in the compute type
  const float *bias;                  // [H * D]
  int H, D, V, R;
  float q_scale, inv_tau;
  int decay;                          // which form turns z into a decay
  int low_tanh, low_f32;              // l passes tanh; l is float whatever the compute type
  const float *bonus;                 // [H, D] or null
};
__device__ __forceinline__ float decay_form(const ChannelIn &a, float z) {
  return a.decay == DECAY_DOUBLE_EXP ? expf(-expf(z)) : decay_of(z, a.inv_tau);
}
template <typename T> __device__ __forceinline__ float low_entry(const ChannelIn &a, size_t t, int r) {
  const float v = a.low_f32 ? ((const float *)a.low)[t * a.low_stride + r] : to_f32(((const T *)a.low)[t * a.low_stride + r]);
  return a.low_tanh ? tanhf(v) : v;
}

// ---------------------------------------------------------------------------
// one token per sequence
// ---------------------------------------------------------------------------
// L lanes hold a column of the state, VEC neighbouring rows at a time (VEC = 4: 16-byte accesses, D a multiple of
// four); a lane takes CS_COLS columns one beside the other so that their loads are in flight together.
#define CS_THREADS 256
#define CS_COLS 4
template <typename T, int VEC, int NR>
__global__ void __launch_bounds__(CS_THREADS)
channel_step_kernel(const ChannelIn a, float *__restrict__ state, const int *__restrict__ seq_slots,
                    float *__restrict__ out, int L) {
  pdl_launch();
  pdl_wait();
  extern __shared__ __align__(16) float cs_sm[];
  const int D = a.D, V = a.V, H = a.H, R = a.R;
  const int Dp = (D + 3) & ~3;
  float *sq = cs_sm, *sk = sq + Dp, *sa = sk + Dp, *low = sa + Dp;
  const int b = blockIdx.z, h = blockIdx.y;
  const int groups = CS_THREADS / L, lane = threadIdx.x % L, group = threadIdx.x / L;
  const int c0 = (blockIdx.x * groups + group) * CS_COLS;
  // the state does not depend on the staged vectors: ask for it first
  float S[CS_COLS][NR][VEC];
  float *sp = state + (((size_t)seq_slots[b] * H + h) * V + c0) * D;
#pragma unroll
  for (int c = 0; c < CS_COLS; ++c)
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      const int d = (r * L + lane) * VEC;
      const bool in = c0 + c < V && d < D;
      if (VEC == 4) {
        const float4 x = in ? *reinterpret_cast<const float4 *>(sp + (size_t)c * D + d) : make_float4(0.f, 0.f, 0.f, 0.f);
        S[c][r][0] = x.x, S[c][r][1 % VEC] = x.y, S[c][r][2 % VEC] = x.z, S[c][r][3 % VEC] = x.w;
      } else {
        S[c][r][0] = in ? sp[(size_t)c * D + d] : 0.f;
      }
    }
  for (int r = threadIdx.x; r < R; r += CS_THREADS) low[r] = low_entry<T>(a, b, r);
  __syncthreads();
  const T *qp = (const T *)a.q + (size_t)b * a.q_stride + (size_t)h * D;
  const T *kp = (const T *)a.k + (size_t)b * a.k_stride + (size_t)h * D;
  for (int d = threadIdx.x; d < Dp; d += CS_THREADS) {
    const bool in = d < D;
    sq[d] = in ? to_f32(qp[d]) * a.q_scale : 0.f;
    sk[d] = in ? to_f32(kp[d]) : 0.f;
    const size_t ch = (size_t)h * D + d;
    sa[d] = in ? decay_form(a, low_dot((const T *)a.w_low + ch * R, low, R, 0.f) + a.bias[ch]) : 0.f;
  }
  __syncthreads();
  float own = 0.f;                                   // what the token's own value counts in its read-out
  const bool bonus = a.bonus;
  if (bonus) {
    __shared__ float scratch[32];
    for (int d = threadIdx.x; d < D; d += CS_THREADS) own = fmaf(sq[d] * sk[d], a.bonus[(size_t)h * D + d], own);
    own = block_sum(own, scratch);
  }
  const T *vp = (const T *)a.v + (size_t)b * a.v_stride + (size_t)h * V;
  float o[CS_COLS];
#pragma unroll
  for (int c = 0; c < CS_COLS; ++c) {
    const float v = c0 + c < V ? to_f32(vp[c0 + c]) : 0.f;
    o[c] = 0.f;
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      const int d = (r * L + lane) * VEC;
      if (d < D) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          const float before = S[c][r][i];
          S[c][r][i] = fmaf(sa[d + i], before, sk[d + i] * v);
          o[c] = fmaf(bonus ? before : S[c][r][i], sq[d + i], o[c]);
        }
        if (c0 + c < V) {
          if (VEC == 4)
            *reinterpret_cast<float4 *>(sp + (size_t)c * D + d) =
                make_float4(S[c][r][0], S[c][r][1 % VEC], S[c][r][2 % VEC], S[c][r][3 % VEC]);
          else
            sp[(size_t)c * D + d] = S[c][r][0];
        }
      }
    }
  }
#pragma unroll
  for (int c = 0; c < CS_COLS; ++c)
    for (int off = L >> 1; off > 0; off >>= 1) o[c] += __shfl_xor_sync(0xffffffffu, o[c], off);
  if (lane == 0) {
#pragma unroll
    for (int c = 0; c < CS_COLS; ++c)
      if (c0 + c < V)
        out[(size_t)b * H * V + (size_t)h * V + c0 + c] = bonus ? fmaf(own, to_f32(vp[c0 + c]), o[c]) : o[c];
  }
}

template <typename T>
static int launch_channel_step(const ChannelIn &a, float *state, const int *seq_slots, int n_seqs, float *out, cudaStream_t stream) {
  const bool vec = a.D % 4 == 0;
  int L = 32;
  if (vec) {
    L = 1;
    while (L < 32 && L * 4 < a.D) L <<= 1;
  }
  const int per_lane = (a.D + L * (vec ? 4 : 1) - 1) / (L * (vec ? 4 : 1));       // at most 4 groups of four, or 16 rows
  const int cols = CS_THREADS / L * CS_COLS;
  const dim3 grid((a.V + cols - 1) / cols, a.H, n_seqs);
  const size_t smem = (size_t)(3 * ((a.D + 3) & ~3) + a.R) * sizeof(float);
  if (vec && per_lane == 1)
    g2b_launch(channel_step_kernel<T, 4, 1>, grid, dim3(CS_THREADS), smem, stream, a, state, seq_slots, out, L);
  else if (vec && per_lane == 2)
    g2b_launch(channel_step_kernel<T, 4, 2>, grid, dim3(CS_THREADS), smem, stream, a, state, seq_slots, out, L);
  else if (vec)
    g2b_launch(channel_step_kernel<T, 4, 4>, grid, dim3(CS_THREADS), smem, stream, a, state, seq_slots, out, L);
  else if (per_lane <= 4)
    g2b_launch(channel_step_kernel<T, 1, 4>, grid, dim3(CS_THREADS), smem, stream, a, state, seq_slots, out, L);
  else
    g2b_launch(channel_step_kernel<T, 1, 16>, grid, dim3(CS_THREADS), smem, stream, a, state, seq_slots, out, L);
  return g2b_check_launch("channel_step");
}

// ---------------------------------------------------------------------------
// prompts: what every column of a head needs of a token, once
// ---------------------------------------------------------------------------
#define CP_TOKENS 8
#define CP_THREADS 128
template <typename T>
__global__ void __launch_bounds__(CP_THREADS)
channel_prep_kernel(const ChannelIn a, int n_tokens, float *__restrict__ qf, float *__restrict__ kf, float *__restrict__ af,
                    float *__restrict__ own) {
  pdl_launch();
  pdl_wait();
  extern __shared__ __align__(16) float cs_sm[];      // low vectors of the block's tokens [CP_TOKENS, R]
  const int D = a.D, R = a.R, h = blockIdx.y;
  const int t0 = blockIdx.x * CP_TOKENS;
  for (int i = threadIdx.x; i < CP_TOKENS * R; i += blockDim.x)       // tokens behind the last one repeat it
    cs_sm[i] = low_entry<T>(a, min(t0 + i / R, n_tokens - 1), i % R);
  __syncthreads();
  const size_t row = (size_t)a.H * D;
  float sum[CP_TOKENS];
#pragma unroll
  for (int i = 0; i < CP_TOKENS; ++i) sum[i] = 0.f;
  for (int d = threadIdx.x; d < D; d += blockDim.x) {
    const size_t ch = (size_t)h * D + d;
    const float u = a.bonus ? a.bonus[ch] : 0.f;
    float z[CP_TOKENS], qv[CP_TOKENS], kv[CP_TOKENS];
#pragma unroll
    for (int i = 0; i < CP_TOKENS; ++i) {
      const size_t t = min(t0 + i, n_tokens - 1);
      qv[i] = to_f32(((const T *)a.q)[t * a.q_stride + ch]);
      kv[i] = to_f32(((const T *)a.k)[t * a.k_stride + ch]);
      z[i] = 0.f;
    }
    const T *w = (const T *)a.w_low + ch * R;
    for (int r = 0; r < R; r += 8)
#pragma unroll
      for (int i = 0; i < CP_TOKENS; ++i) z[i] = low_dot(w + r, cs_sm + i * R + r, 8, z[i]);
    const float bias = a.bias[ch];
#pragma unroll
    for (int i = 0; i < CP_TOKENS; ++i) {
      if (t0 + i >= n_tokens) break;
      const size_t at = (size_t)(t0 + i) * row + ch;
      af[at] = decay_form(a, z[i] + bias);
      qf[at] = qv[i] * a.q_scale;
      kf[at] = kv[i];
      sum[i] = fmaf(qv[i] * a.q_scale * kv[i], u, sum[i]);
    }
  }
  if (!a.bonus) return;
  __shared__ float part[CP_THREADS / 32][CP_TOKENS];
#pragma unroll
  for (int i = 0; i < CP_TOKENS; ++i) {
    const float s = warp_sum(sum[i]);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5][i] = s;
  }
  __syncthreads();
  if (threadIdx.x < CP_TOKENS && t0 + threadIdx.x < n_tokens) {
    float s = 0.f;
    for (int w = 0; w < (int)blockDim.x >> 5; ++w) s += part[w][threadIdx.x];
    own[(size_t)(t0 + threadIdx.x) * a.H + h] = s;
  }
}

// ---------------------------------------------------------------------------
// a segment
// ---------------------------------------------------------------------------
__device__ __forceinline__ void cs_copy16(float *smem, const float *g) {
  const unsigned addr = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(addr), "l"(g));
}

// 128 threads; L lanes hold CC columns, lane l of them the rows 4 (j L + l) .. + 3, j < RG (rows from D on are zeros):
// a row of k, a or q that a lane reads from shared memory serves CC columns, and the lanes of a warp read different
// rows (one warp, one column group, where D is above 64).  Tiles of `tile` tokens (a multiple of four) of k, a (and q)
// as float rows of Dp and of the columns' v, in two buffers: the next tile is on its way while one is computed.
#define SEG_THREADS 128
struct SegArgs {
  const float *qf, *kf, *af;          // [T, H, D]
  const void *v;
  int v_stride, H, D, V;
  const int4 *tiles;                  // (sequence, first row of the step, rows, position)
  int tile_rows;                      // the most rows a tile of the work list has
  const int *seq_meta;                // [B, 4]: first row, rows, tokens before, slot
  float *state;                       // [slots, H, V, D]
  float *seg_state;                   // [segments, H, V, D]: end states, then the states in front
  float *seg_decay;                   // [segments, H, D]: products of the decays
  float *out;                         // [T, H * V]
  const float *own;                   // [T, H] with a bonus: what a token's own value counts in its read-out
  int Dp, tile;
};
// segments of all sequences numbered without gaps that matter: distinct for distinct (sequence, segment)
__device__ __forceinline__ int segment_id(int first_row, int tile_rows, int seq) { return first_row / tile_rows + seq; }

// Sums over L lanes of N values a lane: halves of the values change hands until every lane has N / L of them (or, where
// there are fewer values than lanes, lanes share one); returns the first of the lane's values' index.
template <int N, int L>
__device__ __forceinline__ int lanes_sum(float (&o)[N], int lane) {
  int base = 0, n = N;
#pragma unroll
  for (int m = L >> 1; m > 0; m >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool up = lane & m;
#pragma unroll
      for (int i = 0; i < N / 2; ++i)
        if (i < n) {
          const float send = up ? o[i] : o[i + n], keep = up ? o[i + n] : o[i];
          o[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
        }
      base += up ? n : 0;
    } else {
      o[0] += __shfl_xor_sync(0xffffffffu, o[0], m);
    }
  }
  return base;
}

template <typename T, int L, int RG, int CC, bool READ, bool BONUS>
__global__ void __launch_bounds__(SEG_THREADS)
channel_segment_kernel(const SegArgs a) {
  pdl_launch();
  pdl_wait();
  extern __shared__ __align__(16) float cs_sm[];
  constexpr int COLS = SEG_THREADS / L * CC;
  constexpr int ROWS = READ ? 3 : 2;                 // k, a and, for read-outs, q
  const int4 tl = a.tiles[blockIdx.z];
  const int b = tl.x, first_row = tl.y, n = tl.z;
  const int seq_first = a.seq_meta[4 * b], seq_n = a.seq_meta[4 * b + 1], slot = a.seq_meta[4 * b + 3];
  const bool is_first = first_row == seq_first, is_last = first_row + n == seq_first + seq_n;
  if (!READ && is_last) return;                      // nothing starts behind it: its end state comes with the read-outs
  const int D = a.D, V = a.V, H = a.H, Dp = a.Dp, TT = a.tile;
  const int h = blockIdx.y;
  const int lane = threadIdx.x % L, group = threadIdx.x / L;
  const int c0 = blockIdx.x * COLS + group * CC;
  const int seg = segment_id(first_row, a.tile_rows, b);
  const size_t col_at = ((size_t)h * V + c0) * D;
  float *own = a.seg_state + (size_t)seg * H * V * D + col_at;
  float *slot_state = a.state + (size_t)slot * H * V * D + col_at;
  const int buf_floats = ROWS * TT * Dp;
  float *sv = cs_sm + 2 * buf_floats;                // [2][TT, COLS]
  float *so = sv + 2 * TT * COLS;                    // [2][TT] with a bonus
  const bool vec = (D & 3) == 0;

  float S[CC][RG][4], P[RG][4];
#pragma unroll
  for (int c = 0; c < CC; ++c)
#pragma unroll
    for (int j = 0; j < RG; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = 4 * (j * L + lane) + i;
        float x = 0.f;
        if (READ && c0 + c < V && d < D) x = (is_first && is_last ? slot_state : own)[(size_t)c * D + d];
        S[c][j][i] = x;
        P[j][i] = 1.f;
      }
  for (int i = threadIdx.x; i < 2 * buf_floats; i += SEG_THREADS) cs_sm[i] = 0.f;      // rows from D on stay zero
  __syncthreads();

  const size_t row = (size_t)H * D;
  auto fetch = [&](int t0, int nt, int buf) {
    const size_t at = (size_t)(first_row + t0) * row + (size_t)h * D;
    float *dk = cs_sm + buf * buf_floats, *da = dk + TT * Dp, *dq = da + TT * Dp;
    if (vec) {
      const int per = D >> 2;
      for (int tt = threadIdx.x >> 5; tt < nt; tt += SEG_THREADS / 32)
        for (int p = threadIdx.x & 31; p < per; p += 32) {
          cs_copy16(dk + tt * Dp + 4 * p, a.kf + at + tt * row + 4 * p);
          cs_copy16(da + tt * Dp + 4 * p, a.af + at + tt * row + 4 * p);
          if (READ) cs_copy16(dq + tt * Dp + 4 * p, a.qf + at + tt * row + 4 * p);
        }
    } else {
      for (int i = threadIdx.x; i < nt * D; i += SEG_THREADS) {
        const int tt = i / D, p = i % D;
        dk[tt * Dp + p] = a.kf[at + tt * row + p];
        da[tt * Dp + p] = a.af[at + tt * row + p];
        if (READ) dq[tt * Dp + p] = a.qf[at + tt * row + p];
      }
    }
    asm volatile("cp.async.commit_group;\n" ::);
    // rows that fill the last group of four: they leave the state as it is
    for (int i = threadIdx.x; i < ((nt + 3) / 4 * 4 - nt) * Dp; i += SEG_THREADS) {
      dk[nt * Dp + i] = 0.f;
      da[nt * Dp + i] = 1.f;
    }
    const T *vg = (const T *)a.v + (size_t)(first_row + t0) * a.v_stride + (size_t)h * V + blockIdx.x * COLS;
    float *dv = sv + buf * TT * COLS;
    for (int i = threadIdx.x; i < TT * COLS; i += SEG_THREADS) {
      const int tt = i / COLS, cc = i % COLS;
      dv[i] = tt < nt && blockIdx.x * COLS + cc < V ? to_f32(vg[(size_t)tt * a.v_stride + cc]) : 0.f;
    }
    if (BONUS && threadIdx.x < nt) so[buf * TT + threadIdx.x] = a.own[(size_t)(first_row + t0 + threadIdx.x) * H + h];
  };

  fetch(0, min(TT, n), 0);
  const bool track = !READ && blockIdx.x == 0 && threadIdx.x < 32;     // one warp keeps the decays' products
  int buf = 0;
  for (int t0 = 0; t0 < n; t0 += TT, buf ^= 1) {
    const int nt = min(TT, n - t0);
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();
    if (t0 + TT < n) fetch(t0 + TT, min(TT, n - t0 - TT), buf ^ 1);
    const float *kp = cs_sm + buf * buf_floats + 4 * lane;
    const float *vp = sv + buf * TT * COLS + group * CC;
    for (int u = 0; u < nt; u += 4) {
      float o[4 * CC];
#pragma unroll
      for (int s = 0; s < 4; ++s) {
        const float *k4 = kp + (u + s) * Dp, *a4 = k4 + TT * Dp, *q4 = a4 + TT * Dp;
        float v[CC];
#pragma unroll
        for (int c = 0; c < CC; c += 2) {
          const float2 x = *reinterpret_cast<const float2 *>(vp + (u + s) * COLS + c);
          v[c] = x.x, v[c + 1] = x.y;
        }
#pragma unroll
        for (int c = 0; c < CC; ++c) o[CC * s + c] = 0.f;
#pragma unroll
        for (int j = 0; j < RG; ++j) {
          const float4 kd = *reinterpret_cast<const float4 *>(k4 + 4 * j * L);
          const float4 ad = *reinterpret_cast<const float4 *>(a4 + 4 * j * L);
          float4 qd = make_float4(0.f, 0.f, 0.f, 0.f);
          if (READ) qd = *reinterpret_cast<const float4 *>(q4 + 4 * j * L);
#pragma unroll
          for (int c = 0; c < CC; ++c) {
            if (READ && BONUS)                         // the state in front of the token
              o[CC * s + c] = fmaf(S[c][j][3], qd.w, fmaf(S[c][j][2], qd.z, fmaf(S[c][j][1], qd.y,
                                   fmaf(S[c][j][0], qd.x, o[CC * s + c]))));
            S[c][j][0] = fmaf(ad.x, S[c][j][0], kd.x * v[c]);
            S[c][j][1] = fmaf(ad.y, S[c][j][1], kd.y * v[c]);
            S[c][j][2] = fmaf(ad.z, S[c][j][2], kd.z * v[c]);
            S[c][j][3] = fmaf(ad.w, S[c][j][3], kd.w * v[c]);
            if (READ && !BONUS)
              o[CC * s + c] = fmaf(S[c][j][3], qd.w, fmaf(S[c][j][2], qd.z, fmaf(S[c][j][1], qd.y,
                                   fmaf(S[c][j][0], qd.x, o[CC * s + c]))));
          }
          if (!READ && track) P[j][0] *= ad.x, P[j][1] *= ad.y, P[j][2] *= ad.z, P[j][3] *= ad.w;
        }
      }
      if (READ) {
        constexpr int N = 4 * CC, LEFT = N > L ? N / L : 1;          // values a lane ends with
        const int first = lanes_sum<N, L>(o, lane);
        if (N >= L || lane % (L / (N < L ? N : L)) == 0) {
#pragma unroll
          for (int i = 0; i < LEFT; ++i) {
            const int s = (first + i) / CC, c = (first + i) % CC;
            if (u + s < nt && c0 + c < V) {
              if (BONUS) o[i] = fmaf(so[buf * TT + u + s], vp[(u + s) * COLS + c], o[i]);
              a.out[(size_t)(first_row + t0 + u + s) * H * V + (size_t)h * V + c0 + c] = o[i];
            }
          }
        }
      }
    }
  }
  float *dst = READ ? slot_state : own;
  if (!READ || is_last) {
#pragma unroll
    for (int c = 0; c < CC; ++c)
#pragma unroll
      for (int j = 0; j < RG; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int d = 4 * (j * L + lane) + i;
          if (c0 + c < V && d < D) dst[(size_t)c * D + d] = S[c][j][i];
        }
  }
  if (track && threadIdx.x < L) {
#pragma unroll
    for (int j = 0; j < RG; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = 4 * (j * L + lane) + i;
        if (d < D) a.seg_decay[((size_t)seg * H + h) * D + d] = P[j][i];
      }
  }
}

// The states in front of the segments of a sequence, in place: what a segment left from zero becomes the state
// in front of it.  A thread an entry of the state.
__global__ void __launch_bounds__(256)
channel_carry_kernel(const float *__restrict__ state, float *__restrict__ seg_state, const float *__restrict__ seg_decay,
                     const int *__restrict__ seq_meta, int tile_rows, int H, int D, int V) {
  pdl_launch();
  pdl_wait();
  const int b = blockIdx.y;
  const int first = seq_meta[4 * b], n = seq_meta[4 * b + 1], slot = seq_meta[4 * b + 3];
  const int segs = (n + tile_rows - 1) / tile_rows;
  if (segs <= 1) return;                             // its block reads the slot's state itself
  const int per = H * V * D;
  const int i = blockIdx.x * 256 + threadIdx.x;
  if (i >= per) return;
  const int d = i % D, h = i / (V * D);
  const int id0 = segment_id(first, tile_rows, b);
  float S = state[(size_t)slot * per + i];
  float *e = seg_state + (size_t)id0 * per + i;
  const float *p = seg_decay + ((size_t)id0 * H + h) * D + d;
  // a batch of loads at a time: behind the stores of the places in front, one by one, each would wait for the last
  constexpr int BATCH = 8;
  for (int s0 = 0; s0 < segs; s0 += BATCH) {
    float end[BATCH], dec[BATCH];
#pragma unroll
    for (int j = 0; j < BATCH; ++j) {
      const bool in = s0 + j + 1 < segs;
      end[j] = in ? e[(size_t)(s0 + j) * per] : 0.f;
      dec[j] = in ? p[(size_t)(s0 + j) * H * D] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < BATCH; ++j) {
      if (s0 + j < segs) e[(size_t)(s0 + j) * per] = S;
      S = fmaf(dec[j], S, end[j]);
    }
  }
}

template <typename T, int L, int RG, int CC>
static void launch_segment(const SegArgs &a, int n_tiles, bool read, size_t smem, cudaStream_t stream) {
  constexpr int COLS = SEG_THREADS / L * CC;
  const dim3 grid((a.V + COLS - 1) / COLS, a.H, n_tiles);
  auto kr = a.own ? channel_segment_kernel<T, L, RG, CC, true, true> : channel_segment_kernel<T, L, RG, CC, true, false>;
  auto kw = channel_segment_kernel<T, L, RG, CC, false, false>;
  if (smem > 48 * 1024) cudaFuncSetAttribute(read ? kr : kw, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  g2b_launch(read ? kr : kw, grid, dim3(SEG_THREADS), smem, stream, a);
}

template <typename T>
static int segments(SegArgs a, int n_tiles, bool read, cudaStream_t stream) {
  // rows of the state: 4 a lane on 8, 16 or 32 lanes, or 8, 12 or 16 a lane on 32; 32 entries a lane in all (24 of 12 rows)
  const int L = a.D <= 32 ? 8 : (a.D <= 64 ? 16 : 32);
  const int RG = (a.D + 4 * L - 1) / (4 * L);
  const int CC = RG == 1 ? 8 : (RG == 2 ? 4 : 2);
  a.Dp = RG * 4 * L;
  a.tile = a.Dp <= 128 ? 8 : 4;
  const int cols = SEG_THREADS / L * CC;
  const size_t smem = (size_t)(2 * (read ? 3 : 2) * a.tile * a.Dp + 2 * a.tile * (cols + 1)) * sizeof(float);
#define CS_CASE(L_, RG_, CC_) if (L == L_ && RG == RG_) { launch_segment<T, L_, RG_, CC_>(a, n_tiles, read, smem, stream); return 0; }
  CS_CASE(8, 1, 8) CS_CASE(16, 1, 8) CS_CASE(32, 1, 8) CS_CASE(32, 2, 4) CS_CASE(32, 3, 2) CS_CASE(32, 4, 2)
#undef CS_CASE
  return 1;
}

extern "C" int g2b_channel_scan(int dtype, const void *q, int q_stride, const void *k, int k_stride, const void *v,
                                int v_stride, const void *low, int low_stride, const void *w_low, const float *bias, int H,
                                int D, int V, int R, float q_scale, float inv_tau, int decay, int low_tanh, int low_f32,
                                const float *bonus, float *own, float *state, const int *seq_slots,
                                const int *seq_meta, int n_tokens, int n_seqs, const int *tiles, int n_tiles, int tile_rows,
                                float *qf, float *kf, float *af, float *seg_state, float *seg_decay, float *out,
                                cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return 0;
  if (H <= 0 || V <= 0 || D <= 0 || D > CS_MAX_D) G2B_REFUSE("channel_scan: key size %d outside 1..%d", D, CS_MAX_D);
  if (R <= 0 || R > CS_MAX_R || R % 8) G2B_REFUSE("channel_scan: a decay rank of %d (a multiple of 8 up to %d)", R, CS_MAX_R);
  if ((uintptr_t)w_low & 15) G2B_REFUSE("channel_scan: the decay matrix must start on 16 bytes");
  if (dtype != G2B_F32 && dtype != G2B_BF16) G2B_REFUSE("channel_scan: unknown dtype %d", dtype);
  if (H > 65535 || n_seqs > 65535 || n_tiles > 65535) G2B_REFUSE("channel_scan: %d heads, %d sequences or %d tiles are too many", H, n_seqs, n_tiles);
  if (decay != DECAY_SIGMOID_ROOT && decay != DECAY_DOUBLE_EXP) G2B_REFUSE("channel_scan: unknown form of decay %d", decay);
  ChannelIn in = {q, k, v, low, q_stride, k_stride, v_stride, low_stride, w_low, bias, H, D, V, R, q_scale, inv_tau,
                  decay, low_tanh, low_f32, bonus};
  if (n_tokens == n_seqs)                            // one token per sequence
    return dtype == G2B_F32 ? launch_channel_step<float>(in, state, seq_slots, n_seqs, out, stream)
                            : launch_channel_step<bf16>(in, state, seq_slots, n_seqs, out, stream);
  if (!seq_meta || !tiles || n_tiles <= 0 || tile_rows <= 0 || !qf || !kf || !af || !seg_state || !seg_decay ||
      (bonus && !own))
    G2B_REFUSE("channel_scan: a prompt step needs its tables and scratch buffers");
  const dim3 prep_grid((n_tokens + CP_TOKENS - 1) / CP_TOKENS, H);
  const dim3 prep_block(D > 64 ? CP_THREADS : (D > 32 ? 64 : 32));       // at most a round of idle threads
  const size_t prep_smem = (size_t)CP_TOKENS * R * sizeof(float);
  if (dtype == G2B_F32) {
    if (prep_smem > 48 * 1024) cudaFuncSetAttribute(channel_prep_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)prep_smem);
    g2b_launch(channel_prep_kernel<float>, prep_grid, prep_block, prep_smem, stream, in, n_tokens, qf, kf, af,
               own);
  } else {
    if (prep_smem > 48 * 1024) cudaFuncSetAttribute(channel_prep_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)prep_smem);
    g2b_launch(channel_prep_kernel<bf16>, prep_grid, prep_block, prep_smem, stream, in, n_tokens, qf, kf, af,
               own);
  }
  SegArgs a;
  a.qf = qf; a.kf = kf; a.af = af; a.v = v; a.v_stride = v_stride; a.H = H; a.D = D; a.V = V; a.tiles = (const int4 *)tiles;
  a.tile_rows = tile_rows; a.seq_meta = seq_meta; a.state = state; a.seg_state = seg_state; a.seg_decay = seg_decay; a.out = out;
  a.own = bonus ? own : nullptr;
  a.Dp = a.tile = 0;
  int rc = 0;
  if (n_tiles > n_seqs) {                            // some sequence has several segments
    rc = dtype == G2B_F32 ? segments<float>(a, n_tiles, false, stream) : segments<bf16>(a, n_tiles, false, stream);
    g2b_launch(channel_carry_kernel, dim3((unsigned)(((long long)H * V * D + 255) / 256), n_seqs), dim3(256), 0, stream,
               (const float *)state, seg_state, (const float *)seg_decay, seq_meta, tile_rows, H, D, V);
  }
  rc |= dtype == G2B_F32 ? segments<float>(a, n_tiles, true, stream) : segments<bf16>(a, n_tiles, true, stream);
  if (rc) G2B_REFUSE("channel_scan: no kernel for key size %d", D);
  return g2b_check_launch("channel_scan");
}
