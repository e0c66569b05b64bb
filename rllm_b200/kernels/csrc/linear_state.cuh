// Linear attention with a matrix state per head, the part that both forms of the scan share (linear_state.cu has the
// description): a token's factors from the row of projections [q | k or f | v | (g)].
#pragma once
#include "common.cuh"
#include <math.h>

struct LsArgs {
  int stride, heads, d, dv;      // elements between rows of projections; the head's sizes
  const float* decay;            // fixed decays: [heads]
  const double* inv_freq;        // fixed decays: frequencies of the rotated pairs [rd / 2]
  int rd;
  float k_scale;                 // fixed decays: what a key is multiplied by (behind the rotation)
  const float* f_bias;           // decays per channel: [heads * d]
  const float* lower;            // decays per channel: [heads * d]
  const float* norm_w;           // [dv], or null
  float eps;
  int gated;                     // the row ends in g: the normalised result is multiplied by silu(g)
  const int* positions;
};

__device__ __forceinline__ float ls_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
// sigmoid(z) and sigmoid(-z) = 1 - sigmoid(z), each with its digits, from one exponential
__device__ __forceinline__ void ls_sigmoids(float z, float* pos, float* neg) {
  const float e = expf(-fabsf(z)), r = 1.0f / (1.0f + e), s = e * r;
  *pos = z >= 0.f ? r : s;
  *neg = z >= 0.f ? s : r;
}
__device__ __forceinline__ float ls_silu(float z) { return z / (1.0f + expf(-z)); }

template <typename T>
__device__ __forceinline__ void ls_cos_sin(int pos, double inv_freq, float* c, float* s) {
  if (sizeof(T) == 4) {
    double sd, cd;
    sincos((double)pos * inv_freq, &sd, &cd);
    *c = (float)cd; *s = (float)sd;
  } else {
    rope_cos_sin(pos, inv_freq, c, s);
  }
}
