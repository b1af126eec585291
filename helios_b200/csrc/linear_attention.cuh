// Pieces that the kernels of linear attention share (linear_attention.cu: one fixed decay a head;
// gated_linear_attention.cu: a decay per key channel that depends on the token): sizes of the
// chunked form, vector loads and stores of four neighbours, the state's registers in the kernels
// that walk token by token, the tile product of the chunked form, the gate.
#pragma once
#include "common.cuh"

namespace {

constexpr int LA_C = 64;             // tokens a chunk
constexpr int LA_BLK = 64;           // rows / columns of S a tile
constexpr int LA_LD = LA_BLK + 4;    // row stride of a tile in shared memory (16-byte rows)

template <typename T>
__device__ __forceinline__ void la_load4(const T* p, float (&f)[4]) {
  if constexpr (sizeof(T) == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    f[0] = x.x; f[1] = x.y; f[2] = x.z; f[3] = x.w;
  } else {
    const uint2 x = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  }
}

template <typename T>
__device__ __forceinline__ void la_store4(T* p, const float (&f)[4]) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  }
}

__device__ __forceinline__ float la_gate(float g, int kind) {
  const float s = 1.f / (1.f + expf(-g));
  return kind == 0 ? g * s : s;              // silu | sigmoid
}

constexpr int LA_PARTS = 8;          // warps that share a column's rows
constexpr int LA_STAGE = 8;          // tokens staged in shared memory at a time

template <int VEC>
__device__ __forceinline__ void la_load_state(float (&s)[VEC], const float* p, int left, bool vec) {
  if (VEC == 4 && vec) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    s[0] = x.x;
    if (VEC > 1) s[1 % VEC] = x.y;
    if (VEC > 2) { s[2 % VEC] = x.z; s[3 % VEC] = x.w; }
  } else if (VEC == 2 && vec) {
    const float2 x = *reinterpret_cast<const float2*>(p);
    s[0] = x.x;
    s[1 % VEC] = x.y;
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) s[e] = e < left ? p[e] : 0.f;
  }
}

template <int VEC>
__device__ __forceinline__ void la_store_state(const float (&s)[VEC], float* p, int left, bool vec) {
  if (VEC == 4 && vec) {
    *reinterpret_cast<float4*>(p) = make_float4(s[0], s[1 % VEC], s[2 % VEC], s[3 % VEC]);
  } else if (VEC == 2 && vec) {
    *reinterpret_cast<float2*>(p) = make_float2(s[0], s[1 % VEC]);
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e)
      if (e < left) p[e] = s[e];
  }
}

// q_tiles: (request, first token of the chunk inside the request's step) per chunk of LA_C tokens,
// in the requests' order; a tile at or beyond the request's tokens holds no work.
__device__ __forceinline__ int la_tile_tokens(const int* q_tiles, const int* cu_tokens, int tile, int& tok0) {
  const int seq = q_tiles[2 * tile], l0 = q_tiles[2 * tile + 1];
  const int begin = cu_tokens[seq], n = cu_tokens[seq + 1] - begin;
  if (l0 >= n) return 0;
  tok0 = begin + l0;
  return min(LA_C, n - l0);
}

// acc[i][4 vb + e] += sum_d A[i][d] B[d][64 vb + 4 tx + e] for rows i = ty + 16 r: A [64][LA_LD] rows by
// query token, B [inner][VB * 64 + 4] rows by the inner index.  Four inner steps at a time.  FROM: only
// the row groups r >= FROM.
template <int VB, int FROM = 0>
__device__ __forceinline__ void la_rows_times(float (&acc)[4][4 * VB], const float* A, const float* B, int ty, int tx,
                                              int inner) {
  constexpr int LD = VB * LA_BLK + 4;
#pragma unroll 2
  for (int d = 0; d < inner; d += 4) {
    float x[4][4];
#pragma unroll
    for (int r = FROM; r < 4; ++r) *reinterpret_cast<float4*>(x[r]) = *reinterpret_cast<const float4*>(A + (ty + 16 * r) * LA_LD + d);
#pragma unroll
    for (int u = 0; u < 4; ++u) {
#pragma unroll
      for (int vb = 0; vb < VB; ++vb) {
        const float4 y = *reinterpret_cast<const float4*>(B + (d + u) * LD + vb * LA_BLK + 4 * tx);
#pragma unroll
        for (int r = FROM; r < 4; ++r) {
          acc[r][4 * vb] = fmaf(x[r][u], y.x, acc[r][4 * vb]);
          acc[r][4 * vb + 1] = fmaf(x[r][u], y.y, acc[r][4 * vb + 1]);
          acc[r][4 * vb + 2] = fmaf(x[r][u], y.z, acc[r][4 * vb + 2]);
          acc[r][4 * vb + 3] = fmaf(x[r][u], y.w, acc[r][4 * vb + 3]);
        }
      }
    }
  }
}

}  // namespace
