// Linear attention with ONE fixed decay per head: per head, with q, k [N] and v [M] of a token
// and the head's constant a,
//
//   S <- a S + k v^T        (S is [N, M], float32, carried from token to token in the request's slot)
//   o  = S^T q
//
// q, k and v are columns of a fused projection's rows; on the way in they may pass silu, or q
// and k a rotation of their first `rot` values (value i paired with value i + rot / 2, cos/sin
// tables [T, rot / 2]); k is multiplied by key_scale.  All of that, the recurrence and the
// norms and gates after it are float32.
//
// The decay is a constant, so a stretch of C tokens can be taken at once: with the state S0
// before it,
//   o_i = a^(i+1) S0^T q_i + sum_(j <= i) a^(i-j) (q_i . k_j) v_j
//   S   = a^C S0 + sum_j a^(C-1-j) k_j v_j^T
// Kernels:
//   la_scan       token by token, a block per (request, head, up to 128 columns of S): steps of
//                 few tokens a request; with a norm per head also norm and gate
//   la_chunk_kv   (portions) the sums k_j v_j^T of every chunk of 64 tokens, all chunks in parallel
//   la_states     one pass over a request's chunks: the state before every chunk, and the slot's
//   la_chunk_out  o of every chunk from the state before it and the chunk's own tokens, all
//                 chunks in parallel; with a norm per head also norm and gate
//   la_gate_norm  norm (per head or over the row) times the gate, for what the others leave as
//                 plain float32 o
// The products of the chunked form run on the float32 FMA pipes: the operands are float32 (a
// rotated key, a decayed state), and nothing of the recurrence is rounded to 16 bits.
#include "linear_attention.cuh"

namespace {

enum { LA_NONE = 0, LA_SILU = 1 };

template <typename T>
struct LaIn {
  const T* rows;        // [tokens, ld]
  int ld;
  int q_off, k_off, v_off, g_off;
  const float* cos;     // [tokens, half] or null
  const float* sin;
  int half;
  int act;
  float key_scale;
  int vec;              // four neighbouring columns may be read at once
  int vec_gate;         // ... of the gate, and written to the output
};

__device__ __forceinline__ float la_silu(float x) { return x / (1.f + expf(-x)); }

// Column d of a q or k head (x: the head's first column of the token's row).
template <typename T>
__device__ __forceinline__ float la_qk(const LaIn<T>& in, const T* x, int t, int d) {
  float v = to_float(x[d]);
  if (in.act == LA_SILU) v = la_silu(v);
  if (in.half > 0 && d < 2 * in.half) {
    const int p = d < in.half ? d : d - in.half;
    const float c = in.cos[(size_t)t * in.half + p], s = in.sin[(size_t)t * in.half + p];
    const float o = to_float(x[d < in.half ? d + in.half : d - in.half]);
    v = d < in.half ? v * c - o * s : v * c + o * s;
  }
  return v;
}

// Columns d .. d + 3 of a q or k head (zeros from column N on).
template <typename T>
__device__ __forceinline__ void la_qk4(const LaIn<T>& in, const T* x, int t, int d, int N, float (&f)[4]) {
  if (in.vec && d < N) {          // N, half and all offsets are multiples of 4
    la_load4(x + d, f);
    if (in.act == LA_SILU) {
#pragma unroll
      for (int e = 0; e < 4; ++e) f[e] = la_silu(f[e]);
    }
    if (d < 2 * in.half) {
      const bool lower = d < in.half;
      const int p = lower ? d : d - in.half;
      const float4 c = *reinterpret_cast<const float4*>(in.cos + (size_t)t * in.half + p);
      const float4 s = *reinterpret_cast<const float4*>(in.sin + (size_t)t * in.half + p);
      float o[4];
      la_load4(x + (lower ? d + in.half : d - in.half), o);
      const float sg = lower ? -1.f : 1.f;
      f[0] = f[0] * c.x + sg * o[0] * s.x;
      f[1] = f[1] * c.y + sg * o[1] * s.y;
      f[2] = f[2] * c.z + sg * o[2] * s.z;
      f[3] = f[3] * c.w + sg * o[3] * s.w;
    }
    return;
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) f[e] = d + e < N ? la_qk(in, x, t, d + e) : 0.f;
}

template <typename T>
__device__ __forceinline__ void la_v4(const LaIn<T>& in, const T* x, int d, int M, float (&f)[4]) {
  if (in.vec && d < M) {
    la_load4(x + d, f);
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e) f[e] = d + e < M ? to_float(x[d + e]) : 0.f;
  }
  if (in.act == LA_SILU) {
#pragma unroll
    for (int e = 0; e < 4; ++e) f[e] = la_silu(f[e]);
  }
}

// Pieces of four columns for a thread's B places of a tile of tokens, all loads issued before the
// first use (rows that read four columns at once only: `vec`).  Place b is the token `j[b]` of the
// tile (clamped to a live one) and the columns from d[b] on (clamped to the head's first); `ok[b]`: it is
// a live one, else its values are zeros.
template <int B>
struct LaPlaces {
  int j[B], d[B];
  bool ok[B];
  // i0 + 256 b: place by place, `per_row` pieces of four columns a token, columns from n0 on
  __device__ __forceinline__ LaPlaces(int i0, int per_row, int n0, int n_tok, int N) {
#pragma unroll
    for (int b = 0; b < B; ++b) {
      const int i = i0 + 256 * b, jj = i / per_row, dd = n0 + (i - jj * per_row) * 4;
      ok[b] = jj < n_tok && dd < N;
      j[b] = ok[b] ? jj : 0;
      d[b] = ok[b] ? dd : 0;
    }
  }
};

// The cosines and sines of the places' columns (of columns beyond the rotation: those of the first).
template <typename T, int B>
__device__ __forceinline__ void la_angles(const LaIn<T>& in, int tok0, const LaPlaces<B>& at, float (&c)[B][4],
                                          float (&s)[B][4]) {
#pragma unroll
  for (int b = 0; b < B; ++b) {
    const int d = at.d[b], p = d < in.half ? d : d < 2 * in.half ? d - in.half : 0;
    la_load4(in.cos + (size_t)(tok0 + at.j[b]) * in.half + p, c[b]);
    la_load4(in.sin + (size_t)(tok0 + at.j[b]) * in.half + p, s[b]);
  }
}

// f: the columns as read, o: their partners in the rotation.
template <typename T, int B>
__device__ __forceinline__ void la_fetch(const LaIn<T>& in, const T* x, int tok0, const LaPlaces<B>& at,
                                         float (&f)[B][4], float (&o)[B][4]) {
#pragma unroll
  for (int b = 0; b < B; ++b) {
    const T* r = x + (size_t)(tok0 + at.j[b]) * in.ld;
    const int d = at.d[b];
    la_load4(r + d, f[b]);
    if (in.half > 0) la_load4(r + (d < in.half ? d + in.half : d < 2 * in.half ? d - in.half : d), o[b]);
  }
}

template <typename T, int B>
__device__ __forceinline__ void la_turn(const LaIn<T>& in, const LaPlaces<B>& at, float (&f)[B][4],
                                        const float (&o)[B][4], const float (&c)[B][4], const float (&s)[B][4]) {
#pragma unroll
  for (int b = 0; b < B; ++b) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      if (in.act == LA_SILU) f[b][e] = la_silu(f[b][e]);
      if (in.half > 0 && at.d[b] < 2 * in.half)
        f[b][e] = f[b][e] * c[b][e] + (at.d[b] < in.half ? -o[b][e] : o[b][e]) * s[b][e];
      if (!at.ok[b]) f[b][e] = 0.f;
    }
  }
}

// ---------------------------------------------------------------- token by token
// A warp takes every eighth row of S, a lane VEC neighbouring columns of it, so that whole rows
// of up to 128 columns are read and written at once.  `o` (float32 [T, heads, M]) is written when
// it is given; else (one block a head) norm per head and gate are applied and `out` is written.
template <typename T, int ROWS, int VEC>
__global__ void __launch_bounds__(32 * LA_PARTS)
la_scan_kernel(float* __restrict__ o, T* __restrict__ out, int out_ld, LaIn<T> in, float* __restrict__ state,
               long state_stride, const float* __restrict__ powers, const int* __restrict__ cu_tokens,
               const int* __restrict__ slots, int heads, int N, int M, int vec_state, int gate_kind, float eps,
               float factor) {
  pdl_launch_dependents();
  constexpr int NP = ROWS * LA_PARTS, COLS = 32 * VEC;
  __shared__ float qs[LA_STAGE][NP], ks[LA_STAGE][NP], vs[LA_STAGE][COLS];
  __shared__ float shares[2][LA_PARTS][COLS];
  __shared__ float norm_sums[2][4];
  const int h = blockIdx.y, seq = blockIdx.z;
  const int lane = threadIdx.x & 31, part = threadIdx.x >> 5;
  const int col0 = blockIdx.x * COLS, col = col0 + VEC * lane;
  const int left = M - col;              // live columns from this lane's first on
  const float a = powers[(size_t)h * (LA_C + 1) + 1];
  const int t0 = cu_tokens[seq], t1 = cu_tokens[seq + 1];
  float* S = state + (size_t)slots[seq] * state_stride + (size_t)h * N * M + col;
  pdl_wait();
  float s[ROWS][VEC];
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int n = part + LA_PARTS * i;
    if (n < N && left > 0) la_load_state<VEC>(s[i], S + (size_t)n * M, left, vec_state);
    else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) s[i][e] = 0.f;
    }
  }
  int turn = 0;
  for (int c0 = t0; c0 < t1; c0 += LA_STAGE) {
    const int n_tok = min(LA_STAGE, t1 - c0);
    __syncthreads();
    for (int i = threadIdx.x; i < n_tok * NP; i += blockDim.x) {
      const int j = i / NP, n = i - j * NP;
      const T* r = in.rows + (size_t)(c0 + j) * in.ld + h * N;
      qs[j][n] = n < N ? la_qk(in, r + in.q_off, c0 + j, n) : 0.f;
      ks[j][n] = n < N ? la_qk(in, r + in.k_off, c0 + j, n) * in.key_scale : 0.f;
    }
    for (int i = threadIdx.x; i < n_tok * COLS; i += blockDim.x) {
      const int j = i / COLS, c = i - j * COLS;
      float v = col0 + c < M ? to_float(in.rows[(size_t)(c0 + j) * in.ld + in.v_off + (size_t)h * M + col0 + c]) : 0.f;
      if (in.act == LA_SILU) v = la_silu(v);
      vs[j][c] = v;
    }
    __syncthreads();
    for (int j = 0; j < n_tok; ++j) {
      float v[VEC], acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) { v[e] = vs[j][VEC * lane + e]; acc[e] = 0.f; }
#pragma unroll
      for (int i = 0; i < ROWS; ++i) {
        const int n = part + LA_PARTS * i;
        const float kn = ks[j][n], qn = qs[j][n];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          s[i][e] = fmaf(a, s[i][e], kn * v[e]);
          acc[e] = fmaf(s[i][e], qn, acc[e]);
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) shares[turn][part][VEC * lane + e] = acc[e];
      __syncthreads();
      const int t = c0 + j;
      float r = 0.f;
      if (threadIdx.x < COLS && col0 + threadIdx.x < M) {
#pragma unroll
        for (int p = 0; p < LA_PARTS; ++p) r += shares[turn][p][threadIdx.x];
        if (o != nullptr) o[((size_t)t * heads + h) * M + col0 + threadIdx.x] = r;
      }
      if (o == nullptr) {
        // the head's columns are this block's first warps' threads
        if (threadIdx.x < COLS) {
          const float ss = warp_sum(r * r);
          if (lane == 0) norm_sums[turn][part] = ss;
        }
        __syncthreads();
        if (threadIdx.x < M) {
          float ss = 0.f;
#pragma unroll
          for (int w = 0; w < VEC; ++w) ss += norm_sums[turn][w];
          const float g = to_float(in.rows[(size_t)t * in.ld + in.g_off + (size_t)h * M + threadIdx.x]);
          out[(size_t)t * out_ld + (size_t)h * M + threadIdx.x] =
              from_float<T>(r * factor * rsqrtf(ss / (float)M + eps) * la_gate(g, gate_kind));
        }
      }
      turn ^= 1;
    }
  }
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int n = part + LA_PARTS * i;
    if (n < N && left > 0) la_store_state<VEC>(s[i], S + (size_t)n * M, left, vec_state);
  }
}

// ---------------------------------------------------------------- chunks
// A block takes NB x NB entries of a chunk's sum, a thread E x E of them (NB = 16 E): k_j v_j^T over the
// chunk's tokens from rows in shared memory.
template <typename T, int E>
__global__ void __launch_bounds__(256)
la_chunk_kv_kernel(float* __restrict__ sums, LaIn<T> in, const float* __restrict__ powers,
                   const int* __restrict__ q_tiles, const int* __restrict__ cu_tokens, int heads, int N, int M) {
  pdl_launch_dependents();
  constexpr int NB = 16 * E, LD = NB + 4;
  extern __shared__ __align__(16) float sm[];
  float* Ks = sm;                              // [token][LD]
  float* Vs = sm + LA_C * LD;                  // [token][LD]
  const int tile = blockIdx.x, h = blockIdx.y;
  const int vblocks = (M + NB - 1) / NB;
  const int n0 = (blockIdx.z / vblocks) * NB, m0 = (blockIdx.z % vblocks) * NB;
  int tok0 = 0;
  const int n_tok = la_tile_tokens(q_tiles, cu_tokens, tile, tok0);
  pdl_wait();
  if (n_tok == 0) return;
  const float* pw = powers + (size_t)h * (LA_C + 1);
  if (in.vec) {
    constexpr int B = 4;                     // whole passes: 64 x NB / 4 places are a multiple of 256 B
    static_assert(LA_C * (NB / 4) % (256 * B) == 0, "places of the tile");
    const T* kx = in.rows + in.k_off + (size_t)h * N;
    const T* vx = in.rows + in.v_off + (size_t)h * M;
    for (int i = threadIdx.x; i < n_tok * (NB / 4); i += 256 * B) {
      float f[B][4], o[B][4], c[B][4], sn[B][4], v[B][4];
      const LaPlaces<B> at(i, NB / 4, n0, n_tok, N), av(i, NB / 4, m0, n_tok, M);
      la_fetch(in, kx, tok0, at, f, o);
      if (in.half > 0) la_angles(in, tok0, at, c, sn);
#pragma unroll
      for (int b = 0; b < B; ++b) la_load4(vx + (size_t)(tok0 + av.j[b]) * in.ld + av.d[b], v[b]);
      la_turn(in, at, f, o, c, sn);
#pragma unroll
      for (int b = 0; b < B; ++b) {
        const int p = i + 256 * b, j = p / (NB / 4), d = (p - j * (NB / 4)) * 4;
        if (j >= n_tok) continue;
        const float w = in.key_scale * pw[n_tok - 1 - j];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          if (in.act == LA_SILU) v[b][e] = la_silu(v[b][e]);
          if (!av.ok[b]) v[b][e] = 0.f;
        }
        *reinterpret_cast<float4*>(Ks + j * LD + d) = make_float4(f[b][0] * w, f[b][1] * w, f[b][2] * w, f[b][3] * w);
        *reinterpret_cast<float4*>(Vs + j * LD + d) = make_float4(v[b][0], v[b][1], v[b][2], v[b][3]);
      }
    }
  } else {
    for (int i = threadIdx.x; i < n_tok * (NB / 4); i += 256) {
      const int j = i / (NB / 4), d = (i - j * (NB / 4)) * 4;
      float k4[4], v4[4];
      const T* r = in.rows + (size_t)(tok0 + j) * in.ld;
      la_qk4(in, r + in.k_off + (size_t)h * N, tok0 + j, n0 + d, N, k4);
      la_v4(in, r + in.v_off + (size_t)h * M, m0 + d, M, v4);
      const float f = in.key_scale * pw[n_tok - 1 - j];
      *reinterpret_cast<float4*>(Ks + j * LD + d) = make_float4(k4[0] * f, k4[1] * f, k4[2] * f, k4[3] * f);
      *reinterpret_cast<float4*>(Vs + j * LD + d) = make_float4(v4[0], v4[1], v4[2], v4[3]);
    }
  }
  __syncthreads();
  // rows 4 ty + 64 g + i, columns 4 tx + 64 g' + i': groups of four neighbours, 64 apart
  constexpr int GR = E / 4;
  const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
  float acc[E][E] = {};
#pragma unroll 4
  for (int j = 0; j < n_tok; ++j) {
    float x[E], y[E];
#pragma unroll
    for (int g = 0; g < GR; ++g) {
      *reinterpret_cast<float4*>(x + 4 * g) = *reinterpret_cast<const float4*>(Ks + j * LD + 64 * g + 4 * ty);
      *reinterpret_cast<float4*>(y + 4 * g) = *reinterpret_cast<const float4*>(Vs + j * LD + 64 * g + 4 * tx);
    }
#pragma unroll
    for (int u = 0; u < E; ++u)
#pragma unroll
      for (int w = 0; w < E; ++w) acc[u][w] = fmaf(x[u], y[w], acc[u][w]);
  }
  float* dst = sums + ((size_t)tile * heads + h) * N * M;
#pragma unroll
  for (int u = 0; u < E; ++u) {
    const int n = n0 + 64 * (u / 4) + 4 * ty + u % 4;
    if (n >= N) continue;
#pragma unroll
    for (int g = 0; g < GR; ++g) {
      const int m = m0 + 64 * g + 4 * tx;
      if ((M & 3) == 0) {
        if (m < M)
          *reinterpret_cast<float4*>(dst + (size_t)n * M + m) =
              make_float4(acc[u][4 * g], acc[u][4 * g + 1], acc[u][4 * g + 2], acc[u][4 * g + 3]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (m + e < M) dst[(size_t)n * M + m + e] = acc[u][4 * g + e];
      }
    }
  }
}

// sums[tile] (a chunk's own sum) becomes the state BEFORE the chunk; the slot's state moves on
// to the end of the request's tokens.  A thread W neighbouring entries of S; a request's chunks in
// order.
template <int W>
__global__ void __launch_bounds__(256)
la_states_kernel(float* __restrict__ sums, float* __restrict__ state, long state_stride,
                 const float* __restrict__ powers, const int* __restrict__ cu_tokens,
                 const int* __restrict__ slots, int heads, int NM) {
  pdl_launch_dependents();
  __shared__ int before[8];
  const int h = blockIdx.y, seq = blockIdx.z;
  // chunks of the requests before this one
  int c = 0;
  for (int s = threadIdx.x; s < seq; s += 256) c += (cu_tokens[s + 1] - cu_tokens[s] + LA_C - 1) / LA_C;
  for (int w = 16; w > 0; w >>= 1) c += __shfl_xor_sync(0xffffffffu, c, w);
  if ((threadIdx.x & 31) == 0) before[threadIdx.x >> 5] = c;
  __syncthreads();
  int tile = 0;
  for (int w = 0; w < 8; ++w) tile += before[w];
  const int n = cu_tokens[seq + 1] - cu_tokens[seq];
  const int chunks = (n + LA_C - 1) / LA_C;
  pdl_wait();
  const int e = (blockIdx.x * 256 + threadIdx.x) * W;
  if (e >= NM || chunks == 0) return;
  const float* pw = powers + (size_t)h * (LA_C + 1);
  const float whole = pw[LA_C], rest = pw[n - (chunks - 1) * LA_C];
  float* mine = state + (size_t)slots[seq] * state_stride + (size_t)h * NM + e;
  float s[W];
#pragma unroll
  for (int w = 0; w < W; ++w) s[w] = mine[w];
  const size_t step = (size_t)heads * NM;
  float* u = sums + ((size_t)tile * heads + h) * NM + e;
  constexpr int AHEAD = 8;
  for (int k0 = 0; k0 < chunks; k0 += AHEAD) {
    float v[AHEAD][W];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
      if (k0 + k < chunks) {
        if constexpr (W == 4) la_load4(u + (size_t)(k0 + k) * step, v[k]);
        else v[k][0] = u[(size_t)(k0 + k) * step];
      }
    }
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
      if (k0 + k < chunks) {
        float* dst = u + (size_t)(k0 + k) * step;
        if constexpr (W == 4) la_store4(dst, s);
        else *dst = s[0];
        const float f = k0 + k == chunks - 1 ? rest : whole;
#pragma unroll
        for (int w = 0; w < W; ++w) s[w] = fmaf(f, s[w], v[k][w]);
      }
    }
  }
#pragma unroll
  for (int w = 0; w < W; ++w) mine[w] = s[w];
}

// VB: blocks of 64 columns of v a head has.  A thread owns the query tokens ty + 16 r and, of the
// scores, the key tokens tx + 16 c; of the output, the columns 4 tx + e of every block.  `o`
// (float32 [T, heads, M]) is written when it is given; else the row's norm per head and the gate
// are applied and `out` is written.
template <typename T, int VB>
__global__ void __launch_bounds__(256)
la_chunk_out_kernel(float* __restrict__ o, T* __restrict__ out, int out_ld, LaIn<T> in,
                    const float* __restrict__ states, const float* __restrict__ powers,
                    const int* __restrict__ q_tiles, const int* __restrict__ cu_tokens, int heads, int N, int M,
                    int gate_kind, float eps, float factor) {
  pdl_launch_dependents();
  constexpr int LDB = VB * LA_BLK + 4;
  extern __shared__ __align__(16) float sm[];
  float* Qs = sm;                              // [token][LA_LD]: 64 columns of q, later the scores
  float* Ks = Qs + LA_C * LA_LD;               // [token][LA_LD]: 64 columns of k
  float* Bs = Ks + LA_C * LA_LD;               // 64 rows of S, later of v: [row][LDB]
  float* pw = Bs + LA_BLK * LDB;               // [LA_C + 1]
  const int tile = blockIdx.x, h = blockIdx.y;
  int tok0 = 0;
  const int n_tok = la_tile_tokens(q_tiles, cu_tokens, tile, tok0);
  for (int i = threadIdx.x; i <= LA_C; i += 256) pw[i] = powers[(size_t)h * (LA_C + 1) + i];
  pdl_wait();
  if (n_tok == 0) return;
  const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
  float p[4][4] = {};
  float acc[4][4 * VB] = {};
  const float* S = states + ((size_t)tile * heads + h) * N * M;
  const bool rows16 = (M & 3) == 0;            // rows of S begin at 16-byte boundaries
  for (int n0 = 0; n0 < N; n0 += LA_BLK) {
    if (n0 > 0) __syncthreads();
    const int inner = min(LA_BLK, N - n0);
    // 64 rows of S travel by themselves while q and k are made ready
    for (int i = threadIdx.x; i < LA_BLK * VB * (LA_BLK / 4); i += 256) {
      const int d = i / (VB * (LA_BLK / 4)), m = (i - d * (VB * (LA_BLK / 4))) * 4;
      float* dst = Bs + d * LDB + m;
      if (rows16 && d < inner && m < M) {
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)),
                     "l"(S + (size_t)(n0 + d) * M + m));
      } else {
        float x[4] = {0.f, 0.f, 0.f, 0.f};
        if (d < inner) {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (m + e < M) x[e] = S[(size_t)(n0 + d) * M + m + e];
        }
        *reinterpret_cast<float4*>(dst) = make_float4(x[0], x[1], x[2], x[3]);
      }
    }
    asm volatile("cp.async.commit_group;\n" ::);
    if (in.vec) {
      constexpr int B = 2;
      const T* x = in.rows + (size_t)h * N;
#pragma unroll 1
      for (int i = threadIdx.x; i < LA_C * (LA_BLK / 4); i += 256 * B) {
        float q[B][4], qo[B][4], k[B][4], ko[B][4], c[B][4], sn[B][4];
        const LaPlaces<B> at(i, LA_BLK / 4, n0, n_tok, N);
        la_fetch(in, x + in.q_off, tok0, at, q, qo);
        la_fetch(in, x + in.k_off, tok0, at, k, ko);
        if (in.half > 0) la_angles(in, tok0, at, c, sn);
        la_turn(in, at, q, qo, c, sn);
        la_turn(in, at, k, ko, c, sn);
#pragma unroll
        for (int b = 0; b < B; ++b) {
          const int pl = i + 256 * b, j = pl / (LA_BLK / 4), d = (pl - j * (LA_BLK / 4)) * 4;
          *reinterpret_cast<float4*>(Qs + j * LA_LD + d) = make_float4(q[b][0], q[b][1], q[b][2], q[b][3]);
          *reinterpret_cast<float4*>(Ks + j * LA_LD + d) = make_float4(
              k[b][0] * in.key_scale, k[b][1] * in.key_scale, k[b][2] * in.key_scale, k[b][3] * in.key_scale);
        }
      }
    } else {
      for (int i = threadIdx.x; i < LA_C * (LA_BLK / 4); i += 256) {
        const int j = i / (LA_BLK / 4), d = (i - j * (LA_BLK / 4)) * 4;
        float q4[4] = {0.f, 0.f, 0.f, 0.f}, k4[4] = {0.f, 0.f, 0.f, 0.f};
        if (j < n_tok) {
          const T* r = in.rows + (size_t)(tok0 + j) * in.ld + (size_t)h * N;
          la_qk4(in, r + in.q_off, tok0 + j, n0 + d, N, q4);
          la_qk4(in, r + in.k_off, tok0 + j, n0 + d, N, k4);
        }
        *reinterpret_cast<float4*>(Qs + j * LA_LD + d) = make_float4(q4[0], q4[1], q4[2], q4[3]);
        *reinterpret_cast<float4*>(Ks + j * LA_LD + d) =
            make_float4(k4[0] * in.key_scale, k4[1] * in.key_scale, k4[2] * in.key_scale, k4[3] * in.key_scale);
      }
    }
    asm volatile("cp.async.wait_group 0;\n" ::);
    __syncthreads();
    const int steps = (inner + 3) & ~3;        // zeros beyond `inner`
#pragma unroll 2
    for (int d = 0; d < steps; d += 4) {
      float x[4][4], y[4][4];
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        *reinterpret_cast<float4*>(x[r]) = *reinterpret_cast<const float4*>(Qs + (ty + 16 * r) * LA_LD + d);
        *reinterpret_cast<float4*>(y[r]) = *reinterpret_cast<const float4*>(Ks + (tx + 16 * r) * LA_LD + d);
      }
#pragma unroll
      for (int u = 0; u < 4; ++u)
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j <= i; ++j) p[i][j] = fmaf(x[i][u], y[j][u], p[i][j]);     // later keys are not seen
    }
    la_rows_times<VB>(acc, Qs, Bs, ty, tx, steps);
  }
  // the state's share decays by the tokens since; the chunk's own tokens by their distance
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const float f = pw[ty + 16 * r + 1];
#pragma unroll
    for (int e = 0; e < 4 * VB; ++e) acc[r][e] *= f;
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 4; ++r)
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int dist = ty + 16 * r - (tx + 16 * c);
      Qs[(ty + 16 * r) * LA_LD + tx + 16 * c] = dist >= 0 ? p[r][c] * pw[dist] : 0.f;
    }
  const int key_steps = (n_tok + 3) & ~3;
  if (in.vec) {
    constexpr int B = 4, PER = VB * (LA_BLK / 4);
    const T* vx = in.rows + in.v_off + (size_t)h * M;
    for (int i = threadIdx.x; i < key_steps * PER; i += 256 * B) {
      float v[B][4];
      const LaPlaces<B> at(i, PER, 0, n_tok, M);
#pragma unroll
      for (int b = 0; b < B; ++b) la_load4(vx + (size_t)(tok0 + at.j[b]) * in.ld + at.d[b], v[b]);
#pragma unroll
      for (int b = 0; b < B; ++b) {
        const int pl = i + 256 * b, j = pl / PER, m = (pl - j * PER) * 4;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          if (in.act == LA_SILU) v[b][e] = la_silu(v[b][e]);
          if (!at.ok[b]) v[b][e] = 0.f;
        }
        if (j < key_steps) *reinterpret_cast<float4*>(Bs + j * LDB + m) = make_float4(v[b][0], v[b][1], v[b][2], v[b][3]);
      }
    }
  } else {
    for (int i = threadIdx.x; i < key_steps * VB * (LA_BLK / 4); i += 256) {
      const int j = i / (VB * (LA_BLK / 4)), m = (i - j * (VB * (LA_BLK / 4))) * 4;
      float v4[4] = {0.f, 0.f, 0.f, 0.f};
      if (j < n_tok) la_v4(in, in.rows + (size_t)(tok0 + j) * in.ld + in.v_off + (size_t)h * M, m, M, v4);
      *reinterpret_cast<float4*>(Bs + j * LDB + m) = make_float4(v4[0], v4[1], v4[2], v4[3]);
    }
  }
  __syncthreads();
  // sixteen key tokens at a time, for the query tokens that are not all before them
  la_rows_times<VB, 0>(acc, Qs, Bs, ty, tx, min(16, key_steps));
  if (key_steps > 16) la_rows_times<VB, 1>(acc, Qs + 16, Bs + 16 * LDB, ty, tx, min(16, key_steps - 16));
  if (key_steps > 32) la_rows_times<VB, 2>(acc, Qs + 32, Bs + 32 * LDB, ty, tx, min(16, key_steps - 32));
  if (key_steps > 48) la_rows_times<VB, 3>(acc, Qs + 48, Bs + 48 * LDB, ty, tx, key_steps - 48);
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const int j = ty + 16 * r;
    float ss = 0.f;
    if (o == nullptr) {           // the sixteen threads of a row are neighbouring lanes
#pragma unroll
      for (int e = 0; e < 4 * VB; ++e) ss = fmaf(acc[r][e], acc[r][e], ss);
#pragma unroll
      for (int w = 8; w > 0; w >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
    }
    if (j >= n_tok) continue;
    const int t = tok0 + j;
    const float rstd = factor * rsqrtf(ss / (float)M + eps);
#pragma unroll
    for (int vb = 0; vb < VB; ++vb) {
      const int m = vb * LA_BLK + 4 * tx;
      if (o != nullptr) {
        float* dst = o + ((size_t)t * heads + h) * M + m;
        if (rows16) {
          if (m < M)
            *reinterpret_cast<float4*>(dst) =
                make_float4(acc[r][4 * vb], acc[r][4 * vb + 1], acc[r][4 * vb + 2], acc[r][4 * vb + 3]);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (m + e < M) dst[e] = acc[r][4 * vb + e];
        }
      } else {
        const T* g = in.rows + (size_t)t * in.ld + in.g_off + (size_t)h * M + m;
        T* dst = out + (size_t)t * out_ld + (size_t)h * M + m;
        float g4[4] = {0.f, 0.f, 0.f, 0.f}, y4[4];
        if (in.vec_gate) {
          if (m < M) la_load4(g, g4);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (m + e < M) g4[e] = to_float(g[e]);
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) y4[e] = acc[r][4 * vb + e] * rstd * la_gate(g4[e], gate_kind);
        if (in.vec_gate) {
          if (m < M) la_store4(dst, y4);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (m + e < M) dst[e] = from_float<T>(y4[e]);
        }
      }
    }
  }
}

// ---------------------------------------------------------------- norm and gate
// out = factor * o / rms(o) (* weight) * gate(g): per head (a block a (token, head)) or over the
// row (a block a token); the weight has an entry per value of the norm.
template <typename T>
__global__ void la_gate_norm_kernel(T* __restrict__ out, int out_ld, const float* __restrict__ o,
                                    const T* __restrict__ gate, int gate_ld, const float* __restrict__ weight,
                                    int parts, int width, int gate_kind, float eps, float factor) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float scratch[33];
  const int t = blockIdx.x / parts, part = blockIdx.x - t * parts;
  const float* x = o + (size_t)blockIdx.x * width;
  float ss = 0.f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) ss = fmaf(x[c], x[c], ss);
  const float rstd = factor * rsqrtf(block_sum(ss, scratch) / (float)width + eps);
  const T* g = gate + (size_t)t * gate_ld + (size_t)part * width;
  T* y = out + (size_t)t * out_ld + (size_t)part * width;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    float v = x[c] * rstd * la_gate(to_float(g[c]), gate_kind);
    if (weight) v *= weight[c];
    y[c] = from_float<T>(v);
  }
}

// The same with four neighbouring values at a time and the row held in registers between the
// passes: widths that are multiples of 4 up to 4 x 256 x GROUPS.
template <typename T, int GROUPS>
__global__ void __launch_bounds__(256)
la_gate_norm_vec_kernel(T* __restrict__ out, int out_ld, const float* __restrict__ o, const T* __restrict__ gate,
                        int gate_ld, const float* __restrict__ weight, int parts, int width, int gate_kind, float eps,
                        float factor) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float scratch[33];
  const int t = blockIdx.x / parts, part = blockIdx.x - t * parts;
  const float* x = o + (size_t)blockIdx.x * width;
  const T* g = gate + (size_t)t * gate_ld + (size_t)part * width;
  T* y = out + (size_t)t * out_ld + (size_t)part * width;
  float v[GROUPS][4], gv[GROUPS][4];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < GROUPS; ++k) {
    const int c = (k * blockDim.x + threadIdx.x) * 4;
    if (c < width) {
      la_load4(x + c, v[k]);
      la_load4(g + c, gv[k]);
    }
  }
#pragma unroll
  for (int k = 0; k < GROUPS; ++k) {
    if ((k * blockDim.x + threadIdx.x) * 4 < width) {
#pragma unroll
      for (int e = 0; e < 4; ++e) ss = fmaf(v[k][e], v[k][e], ss);
    }
  }
  const float rstd = factor * rsqrtf(block_sum(ss, scratch) / (float)width + eps);
#pragma unroll
  for (int k = 0; k < GROUPS; ++k) {
    const int c = (k * blockDim.x + threadIdx.x) * 4;
    if (c < width) {
      float w[4] = {1.f, 1.f, 1.f, 1.f};
      if (weight) la_load4(weight + c, w);
#pragma unroll
      for (int e = 0; e < 4; ++e) v[k][e] *= rstd * w[e] * la_gate(gv[k][e], gate_kind);
      la_store4(y + c, v[k]);
    }
  }
}

template <typename T>
LaIn<T> la_in(const void* rows, int ld, int q_off, int k_off, int v_off, int g_off, const float* cos,
              const float* sin, int rot, int act, float key_scale, int N, int M) {
  LaIn<T> in;
  in.rows = (const T*)rows; in.ld = ld;
  in.q_off = q_off; in.k_off = k_off; in.v_off = v_off; in.g_off = g_off;
  in.cos = cos; in.sin = sin; in.half = cos ? rot / 2 : 0;
  in.act = act; in.key_scale = key_scale;
  in.vec = ((ld | q_off | k_off | v_off | N | M | in.half) & 3) == 0 && ((uintptr_t)rows & 15) == 0 &&
           ((uintptr_t)cos & 15) == 0 && ((uintptr_t)sin & 15) == 0;
  in.vec_gate = 0;
  return in;
}

template <typename T, int VB>
int la_launch_out(float* o, T* out, int out_ld, const LaIn<T>& in, const float* states, const float* powers,
                  const int* q_tiles, int n_tiles, const int* cu_tokens, int heads, int N, int M, int gate_kind,
                  float eps, float factor, cudaStream_t stream) {
  constexpr size_t SMEM = (2 * LA_C * LA_LD + LA_BLK * (VB * LA_BLK + 4) + LA_C + 1) * sizeof(float);
  auto kernel = la_chunk_out_kernel<T, VB>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM) != cudaSuccess)
      return HB_LAUNCH_FAILED;
    configured = true;
  }
  hb_launch(kernel, dim3(n_tiles, heads), dim3(256), SMEM, stream, o, out, out_ld, in, states, powers, q_tiles,
            cu_tokens, heads, N, M, gate_kind, eps, factor);
  return hb_check_launch();
}

template <typename T, int E>
int la_launch_kv(float* sums, const LaIn<T>& in, const float* powers, const int* q_tiles, int n_tiles,
                 const int* cu_tokens, int heads, int N, int M, cudaStream_t stream) {
  constexpr int NB = 16 * E;
  constexpr size_t SMEM = 2 * LA_C * (NB + 4) * sizeof(float);
  auto kernel = la_chunk_kv_kernel<T, E>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM) != cudaSuccess)
      return HB_LAUNCH_FAILED;
    configured = true;
  }
  hb_launch(kernel, dim3(n_tiles, heads, ((N + NB - 1) / NB) * ((M + NB - 1) / NB)), dim3(256), SMEM, stream, sums, in,
            powers, q_tiles, cu_tokens, heads, N, M);
  return hb_check_launch();
}

}  // namespace

// rows [T, ld]: q, k (heads x N), v and the gate (heads x M) at the given columns.  powers
// [heads, 65]: the decay to the power 0..64.  `o` null (M <= 128): norm per head and gate are
// applied and `out` (rows out_ld apart) is written; else o [T, heads, M] float32.
HB_EXPORT int hb_la_scan(float* o, void* out, int out_ld, const void* rows, int ld, int q_off, int k_off, int v_off,
                         int g_off, const float* cos, const float* sin, int rot, int act, float key_scale,
                         float* state, long state_stride, const float* powers, const int* cu_tokens,
                         const int* slots, int T, int S, int heads, int N, int M, int gate_kind, float eps,
                         float factor, int act_dt, cudaStream_t stream) {
  if (T <= 0 || S <= 0) return HB_OK;
  if (N <= 0 || N > 256 || M <= 0 || heads <= 0 || (o == nullptr && M > 128)) return HB_BAD_ARGUMENT;
  const int vec = M <= 32 ? 1 : M <= 64 ? 2 : 4;
  const dim3 grid((M + 32 * vec - 1) / (32 * vec), heads, S);
  const int vec_state = M % vec == 0 && state_stride % vec == 0 && ((uintptr_t)state & (4 * vec - 1)) == 0;
#define HB_LA_SCAN(TA, R, V)                                                                                \
  hb_launch(la_scan_kernel<TA, R, V>, grid, dim3(32 * LA_PARTS), 0, stream, o, (TA*)out, out_ld,              \
            la_in<TA>(rows, ld, q_off, k_off, v_off, g_off, cos, sin, rot, act, key_scale, N, M), state,      \
            state_stride, powers, cu_tokens, slots, heads, N, M, vec_state, gate_kind, eps, factor)
#define HB_LA_SCAN_V(TA, V)                                                                                 \
  do {                                                                                                       \
    if (N <= 32) HB_LA_SCAN(TA, 4, V);                                                                       \
    else if (N <= 64) HB_LA_SCAN(TA, 8, V);                                                                  \
    else if (N <= 128) HB_LA_SCAN(TA, 16, V);                                                                \
    else HB_LA_SCAN(TA, 32, V);                                                                              \
  } while (0)
  HB_DISPATCH_DTYPE(act_dt, TA,
    if (vec == 1) HB_LA_SCAN_V(TA, 1);
    else if (vec == 2) HB_LA_SCAN_V(TA, 2);
    else HB_LA_SCAN_V(TA, 4));
#undef HB_LA_SCAN_V
#undef HB_LA_SCAN
  return hb_check_launch();
}

// Chunked: sums [tiles, heads, N, M] float32 is scratch.  `o` null: norm per head and gate are
// applied and `out` (rows out_ld apart) is written; else o [T, heads, M] float32.
HB_EXPORT int hb_la_chunked(float* o, void* out, int out_ld, float* sums, const void* rows, int ld, int q_off,
                            int k_off, int v_off, int g_off, const float* cos, const float* sin, int rot, int act,
                            float key_scale, float* state, long state_stride, const float* powers,
                            const int* q_tiles, int n_tiles, const int* cu_tokens, const int* slots, int S, int heads,
                            int N, int M, int gate_kind, float eps, float factor, int act_dt, cudaStream_t stream) {
  if (n_tiles <= 0 || S <= 0) return HB_OK;
  if (N <= 0 || N > 256 || M <= 0 || M > 256 || heads <= 0 || ((uintptr_t)sums & 15)) return HB_BAD_ARGUMENT;
  HB_DISPATCH_DTYPE(act_dt, TA, {
    LaIn<TA> in = la_in<TA>(rows, ld, q_off, k_off, v_off, g_off, cos, sin, rot, act, key_scale, N, M);
    in.vec_gate = ((ld | g_off | M | out_ld) & 3) == 0 && (((uintptr_t)rows | (uintptr_t)out) & 15) == 0;
    int st = N > 64 || M > 64 ? la_launch_kv<TA, 8>(sums, in, powers, q_tiles, n_tiles, cu_tokens, heads, N, M, stream)
                              : la_launch_kv<TA, 4>(sums, in, powers, q_tiles, n_tiles, cu_tokens, heads, N, M, stream);
    if (st != HB_OK) return st;
    const int NM = N * M;
    if (NM % 4 == 0)
      hb_launch(la_states_kernel<4>, dim3((NM / 4 + 255) / 256, heads, S), dim3(256), 0, stream, sums, state,
                state_stride, powers, cu_tokens, slots, heads, NM);
    else
      hb_launch(la_states_kernel<1>, dim3((NM + 255) / 256, heads, S), dim3(256), 0, stream, sums, state, state_stride,
                powers, cu_tokens, slots, heads, NM);
    const int vb = (M + LA_BLK - 1) / LA_BLK;
    if (vb == 1) st = la_launch_out<TA, 1>(o, (TA*)out, out_ld, in, sums, powers, q_tiles, n_tiles, cu_tokens, heads, N, M, gate_kind, eps, factor, stream);
    else if (vb == 2) st = la_launch_out<TA, 2>(o, (TA*)out, out_ld, in, sums, powers, q_tiles, n_tiles, cu_tokens, heads, N, M, gate_kind, eps, factor, stream);
    else st = la_launch_out<TA, 4>(o, (TA*)out, out_ld, in, sums, powers, q_tiles, n_tiles, cu_tokens, heads, N, M, gate_kind, eps, factor, stream);
    return st;
  });
  return HB_OK;
}

// parts: norms a row has (heads: per head, 1: over the row), each `width` values wide; weight
// [width] (or null): one for all of them.
HB_EXPORT int hb_la_gate_norm(void* out, int out_ld, const float* o, const void* gate, int gate_ld,
                              const float* weight, int T, int parts, int width, int gate_kind, float eps,
                              float factor, int act_dt, cudaStream_t stream) {
  if (T <= 0) return HB_OK;
  if (parts <= 0 || width <= 0) return HB_BAD_ARGUMENT;
  int threads = 32;
  if (width % 4 == 0 && width <= 4096 && ((gate_ld | out_ld) & 3) == 0 &&
      (((uintptr_t)out | (uintptr_t)o | (uintptr_t)weight) & 15) == 0 &&
      ((uintptr_t)gate & (act_dt == HB_F32 ? 15 : 7)) == 0) {
    while (threads < 256 && threads * 4 < width) threads *= 2;
    const int groups = (width + 4 * threads - 1) / (4 * threads);
#define HB_GATE_NORM(G)                                                                                       \
    hb_launch(la_gate_norm_vec_kernel<TA, G>, dim3((unsigned)(T * parts)), dim3(threads), 0, stream, (TA*)out,  \
              out_ld, o, (const TA*)gate, gate_ld, weight, parts, width, gate_kind, eps, factor)
    HB_DISPATCH_DTYPE(act_dt, TA,
      if (groups == 1) HB_GATE_NORM(1);
      else if (groups == 2) HB_GATE_NORM(2);
      else HB_GATE_NORM(4));
#undef HB_GATE_NORM
    return hb_check_launch();
  }
  while (threads < 256 && threads * 2 < width) threads *= 2;
  HB_DISPATCH_DTYPE(act_dt, TA,
    hb_launch(la_gate_norm_kernel<TA>, dim3((unsigned)(T * parts)), dim3(threads), 0, stream, (TA*)out, out_ld, o,
              (const TA*)gate, gate_ld, weight, parts, width, gate_kind, eps, factor));
  return hb_check_launch();
}
