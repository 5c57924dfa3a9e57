// The result of routed experts before it is added up: token t's row is the sum over its slots s, in slot order, of
// weights[t, s] (or 1) times row row_of_pair[t * top + s] (or t * top + s) of y, itself the sum of `n_parts` unsummed
// parts in ascending order.  All fp32.
#pragma once
#include "common.cuh"

struct RowSum {
  const float* y;                // null: there is none
  int n_parts;
  int64_t part_stride;
  const int* row_of_pair;
  const float* weights;
  int top;

  // columns c .. c + VEC - 1 of token t (VEC 4: 16-byte aligned); the rows of four slots are requested together
  template <int VEC> __device__ __forceinline__ void sum(int64_t t, int c, int width, float (&acc)[VEC]) const {
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
    for (int s0 = 0; s0 < top; s0 += 4) {
      float v[4][VEC];
#pragma unroll
      for (int q = 0; q < 4; ++q) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[q][e] = 0.f;
        if (s0 + q < top) {
          const int64_t row = row_of_pair ? (int64_t)row_of_pair[t * top + s0 + q] : t * top + s0 + q;
          const float* p = y + row * width + c;
          for (int k = 0; k < n_parts; ++k, p += part_stride) {
            if (VEC == 4) {
              const float4 x = __ldcg(reinterpret_cast<const float4*>(p));
              v[q][0] += x.x, v[q][VEC > 1 ? 1 : 0] += x.y, v[q][VEC > 2 ? 2 : 0] += x.z, v[q][VEC > 3 ? 3 : 0] += x.w;
            } else {
              v[q][0] += __ldcg(p);
            }
          }
        }
      }
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        if (s0 + q >= top) break;
        const float w = weights ? weights[t * top + s0 + q] : 1.f;
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = fmaf(w, v[q][e], acc[e]);
      }
    }
  }
};
