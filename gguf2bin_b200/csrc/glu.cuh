// The gate of a feed-forward with two input matrices, in one form with four numbers:
//   out = g * sigmoid(g (c1 + c3 g^2)) * (u + offset),  g = min(gate, limit),  u = clamp(up, -limit, limit)
// SiLU: limit infinite, offset 0, c1 1, c3 0.  The tanh form of GELU, 0.5 z (1 + tanh(k (z + 0.044715 z^3)))
// with k = sqrt(2/pi), is z * sigmoid(2 k (z + 0.044715 z^3)): c1 = 2 k, c3 = 0.044715 c1.  The capped gate:
// its limit, offset 1, c1 its slope.
#pragma once

struct GluForm {
  float limit, offset, c1, c3;
};

__device__ __forceinline__ float glu_value(float gate, float up, const GluForm &f) {
  const float g = fminf(gate, f.limit);
  const float u = fminf(fmaxf(up, -f.limit), f.limit) + f.offset;
  return g / (1.f + expf(-(g * fmaf(f.c3 * g, g, f.c1)))) * u;
}

// The same from the fast exponential and division, for epilogues that round to bfloat16.
__device__ __forceinline__ float glu_value_fast(float gate, float up, const GluForm &f) {
  const float g = fminf(gate, f.limit);
  const float u = fminf(fmaxf(up, -f.limit), f.limit) + f.offset;
  return __fdividef(g, 1.f + __expf(-(g * fmaf(f.c3 * g, g, f.c1)))) * u;
}

// The activation alone: z * sigmoid(z (c1 + c3 z^2)).
__device__ __forceinline__ float act_value(float z, const GluForm &f) { return z / (1.f + expf(-(z * fmaf(f.c3 * z, z, f.c1)))); }
__device__ __forceinline__ float act_value_fast(float z, const GluForm &f) {
  return __fdividef(z, 1.f + __expf(-(z * fmaf(f.c3 * z, z, f.c1))));
}

// What a product's kernel gets beside its operands: the form of its epilogue, and, where the columns of C come from
// several inputs (W's rows in groups of `a_group`, A a stack of as many [M, K] matrices), the size of a group; 0: one A.
struct ProductTail : GluForm {
  int a_group;
  // the first row of the A that the columns from n0 on are a product of
  __device__ __forceinline__ int a_row(int n0, int M) const { return a_group ? n0 / a_group * M : 0; }
};
