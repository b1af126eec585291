// Linear attention whose decay is a vector that depends on the token: per head, with q, k [N], v [M]
// and the decay a [N] (one per key channel) of a token,
//
//   S <- diag(a) S + k v^T      (S is [N, M], float32, carried from token to token in the request's slot)
//   o  = S^T q
//   a  = sigmoid(z)^(1 / tau),   z = W2 (low-rank columns of the token's row) + bias
//
// q, k, v, the low-rank columns and the gate are columns of one fused projection's rows; q is
// multiplied by q_scale.  o is normed per head (a weight per value, shared by the heads) and
// multiplied by silu(gate) and a constant factor.  The product with W2, the decays, the recurrence, the norm and the gate
// are float32.
//
// A stretch of tokens can be taken at once.  With P(j, i] the product of the decays after token j up
// to i, channel by channel, and S0 the state before the stretch,
//   o_i = S0^T (P(-1, i] q_i) + sum_(j <= i) (sum_n q_in P(j, i]_n k_jn) v_j
//   S   = diag(P(-1, last]) S0 + sum_j (P(j, last] k_j) v_j^T
// Only products of decays over runs of tokens are formed, never quotients or exponentials of
// differences: nothing overflows, and a product that underflows is a contribution that is 0.
// A chunk of 64 tokens is cut into four sub-chunks of 16:
//   Q_i = q_i times the decays from its sub-chunk's start to i, K_j = k_j times those after j to its
//   sub-chunk's end, D_s the product over sub-chunk s; a pair of tokens in different sub-chunks meets
//   as Q_i . (D between them) K_j, a pair in the same one with the running product itself.
// Kernels:
//   gla_scan       token by token, a block per (request, head, up to 128 columns of S): steps of few
//                  tokens a request; with one block a head also norm and gate
//   gla_prepare    (portions) decays, Q, K, D and the scores of pairs inside a sub-chunk
//   gla_chunk_kv   every chunk's own sum of k v^T
//   gla_states     one pass over a request's chunks: the state before every chunk, and the slot's
//   gla_chunk_out  o of every chunk, norm and gate
// The products run on the float32 FMA pipes: their operands are float32.
#include "linear_attention.cuh"

namespace {

constexpr int GLA_SUB = 16;                  // tokens a sub-chunk
constexpr int GLA_SUBS = LA_C / GLA_SUB;
static_assert(GLA_SUBS == 4, "the kernels pair a thread's rows 16 apart with the sub-chunks");

template <typename T>
struct GlaIn {
  const T* rows;        // [tokens, ld]
  int ld;
  int q_off, k_off, v_off, g_off, a_off;
  const T* w2;          // [heads * N, R]
  const float* bias;    // [heads * N]
  int R;
  float inv_tau, q_scale;
  int vec;              // four neighbouring columns of v may be read at once
  int vec_gate;         // ... of the gate, and written to the output
  int vec_w2;           // ... of W2's rows
};

// sigmoid(z)^(1 / tau)
__device__ __forceinline__ float gla_decay(float z, float inv_tau) {
  return expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau);
}

// Four neighbouring values from column d of `left` live ones on, zeros beyond.
template <typename T>
__device__ __forceinline__ void gla_load4(const T* p, int left, bool vec, float (&f)[4]) {
  if (vec && left > 0) {
    la_load4(p, f);
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e) f[e] = e < left ? to_float(p[e]) : 0.f;
  }
}

// ---------------------------------------------------------------- token by token
// A warp takes every eighth row of S, a lane VEC neighbouring columns of it.  `o` (float32 [T, heads,
// M]) is written when it is given; else (one block a head) norm and gate are applied and `out` is.
template <typename T, int ROWS, int VEC>
__global__ void __launch_bounds__(32 * LA_PARTS)
gla_scan_kernel(float* __restrict__ o, T* __restrict__ out, int out_ld, GlaIn<T> in, float* __restrict__ state,
                long state_stride, const int* __restrict__ cu_tokens, const int* __restrict__ slots, int heads, int N,
                int M, int vec_state, const float* __restrict__ norm_weight, float eps, float factor) {
  pdl_launch_dependents();
  constexpr int NP = ROWS * LA_PARTS, COLS = 32 * VEC;
  __shared__ float qs[LA_STAGE][NP], ks[LA_STAGE][NP], as[LA_STAGE][NP], vs[LA_STAGE][COLS];
  __shared__ float shares[2][LA_PARTS][COLS];
  __shared__ float norm_sums[2][4];
  const int h = blockIdx.y, seq = blockIdx.z;
  const int lane = threadIdx.x & 31, part = threadIdx.x >> 5;
  const int col0 = blockIdx.x * COLS, col = col0 + VEC * lane;
  const int left = M - col;              // live columns from this lane's first on
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
      const T* r = in.rows + (size_t)(c0 + j) * in.ld;
      const bool live = n < N;
      const int c = h * N + (live ? n : 0);
      qs[j][n] = live ? to_float(r[in.q_off + c]) * in.q_scale : 0.f;
      ks[j][n] = live ? to_float(r[in.k_off + c]) : 0.f;
      float z = in.bias[c];
      const T* w = in.w2 + (size_t)c * in.R;
      const T* a = r + in.a_off;
      if (in.vec_w2) {
#pragma unroll 4
        for (int e = 0; e < in.R; e += 4) {
          float w4[4];
          la_load4(w + e, w4);
#pragma unroll
          for (int u = 0; u < 4; ++u) z = fmaf(w4[u], to_float(a[e + u]), z);
        }
      } else {
        for (int e = 0; e < in.R; ++e) z = fmaf(to_float(w[e]), to_float(a[e]), z);
      }
      as[j][n] = live ? gla_decay(z, in.inv_tau) : 0.f;
    }
    for (int i = threadIdx.x; i < n_tok * COLS; i += blockDim.x) {
      const int j = i / COLS, c = i - j * COLS;
      vs[j][c] = col0 + c < M ? to_float(in.rows[(size_t)(c0 + j) * in.ld + in.v_off + (size_t)h * M + col0 + c]) : 0.f;
    }
    __syncthreads();
    for (int j = 0; j < n_tok; ++j) {
      float v[VEC], acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) { v[e] = vs[j][VEC * lane + e]; acc[e] = 0.f; }
#pragma unroll
      for (int i = 0; i < ROWS; ++i) {
        const int n = part + LA_PARTS * i;
        const float an = as[j][n], kn = ks[j][n], qn = qs[j][n];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          s[i][e] = fmaf(an, s[i][e], kn * v[e]);
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
              from_float<T>(r * factor * rsqrtf(ss / (float)M + eps) * norm_weight[threadIdx.x] * la_gate(g, 0));
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
// A block a (chunk, head), 64 key channels at a time.  First a thread is (channel, sub-chunk): its
// sixteen decays, and the running products along them, stay in registers.  Then it is (four
// channels, four key tokens, sub-chunk) for the scores of pairs inside a sub-chunk.
//   Q, K   float [T, heads, N]
//   D      float [tiles, heads, 5, N]: the product of the decays over every sub-chunk, then over the chunk
//   diag   float [tiles, heads, 64, 16]: query token of the chunk x key token of the same sub-chunk
template <typename T>
__global__ void __launch_bounds__(256, 2)
gla_prepare_kernel(float* __restrict__ Q, float* __restrict__ K, float* __restrict__ D, float* __restrict__ diag,
                   GlaIn<T> in, const int* __restrict__ q_tiles, const int* __restrict__ cu_tokens, int heads, int N) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float sm[];
  float* qs = sm;                              // [token][LA_LD]
  float* ks = qs + LA_C * LA_LD;
  float* as = ks + LA_C * LA_LD;
  float* tot = as + LA_C * LA_LD;              // [sub-chunk][64]
  float* low = tot + GLA_SUBS * LA_BLK;        // [token][R rounded up to 4]
  const int tile = blockIdx.x, h = blockIdx.y;
  int tok0 = 0;
  const int n_tok = la_tile_tokens(q_tiles, cu_tokens, tile, tok0);
  const int RL = (in.R + 3) & ~3;
  pdl_wait();
  if (n_tok == 0) return;
  for (int i = threadIdx.x; i < LA_C * RL; i += 256) {
    const int j = i / RL, r = i - j * RL;
    low[i] = j < n_tok && r < in.R ? to_float(in.rows[(size_t)(tok0 + j) * in.ld + in.a_off + r]) : 0.f;
  }
  __syncthreads();
  const int d = threadIdx.x & 63, sub = threadIdx.x >> 6;
  const int sl = threadIdx.x & 15, jq = (threadIdx.x >> 4) & 3;      // (the sub-chunk is `sub` again)
  float p[4][GLA_SUB];
#pragma unroll
  for (int a = 0; a < 4; ++a)
#pragma unroll
    for (int i = 0; i < GLA_SUB; ++i) p[a][i] = 0.f;
  for (int n0 = 0; n0 < N; n0 += LA_BLK) {
    const int n = n0 + d;
    const bool live = n < N;
    const int c = h * N + (live ? n : 0);
    if (n0 > 0) __syncthreads();
    {
      float qv[GLA_SUB], kv[GLA_SUB];
#pragma unroll
      for (int i = 0; i < GLA_SUB; ++i) {
        const int j = sub * GLA_SUB + i;
        const T* r = in.rows + (size_t)(tok0 + (j < n_tok ? j : 0)) * in.ld + c;
        qv[i] = to_float(r[in.q_off]);
        kv[i] = to_float(r[in.k_off]);
      }
#pragma unroll
      for (int i = 0; i < GLA_SUB; ++i) {
        const int j = sub * GLA_SUB + i;
        const bool ok = live && j < n_tok;
        qs[j * LA_LD + d] = ok ? qv[i] * in.q_scale : 0.f;
        ks[j * LA_LD + d] = ok ? kv[i] : 0.f;
      }
    }
    float z[GLA_SUB];
    const float b = in.bias[c];
#pragma unroll
    for (int i = 0; i < GLA_SUB; ++i) z[i] = b;
    const T* w = in.w2 + (size_t)c * in.R;
    for (int r = 0; r < in.R; r += 4) {
      float w4[4];
      gla_load4(w + r, in.R - r, in.vec_w2, w4);
#pragma unroll
      for (int i = 0; i < GLA_SUB; ++i) {
        const float4 a = *reinterpret_cast<const float4*>(low + (size_t)(sub * GLA_SUB + i) * RL + r);
        z[i] = fmaf(w4[0], a.x, z[i]);
        z[i] = fmaf(w4[1], a.y, z[i]);
        z[i] = fmaf(w4[2], a.z, z[i]);
        z[i] = fmaf(w4[3], a.w, z[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < GLA_SUB; ++i) {
      const int j = sub * GLA_SUB + i;
      z[i] = live && j < n_tok ? gla_decay(z[i], in.inv_tau) : 1.f;
      as[j * LA_LD + d] = z[i];
    }
    // (a thread reads back the q and k that it wrote itself)
    float* Dc = D + ((size_t)tile * heads + h) * 5 * N;
    const size_t at0 = (size_t)(tok0 + sub * GLA_SUB) * heads * N + c, step = (size_t)heads * N;
    const int own = live ? n_tok - sub * GLA_SUB : 0;            // live tokens of the sub-chunk
    float run = 1.f;
#pragma unroll
    for (int i = 0; i < GLA_SUB; ++i) {
      run *= z[i];
      if (i < own) Q[at0 + i * step] = qs[(sub * GLA_SUB + i) * LA_LD + d] * run;
    }
    tot[sub * LA_BLK + d] = run;
    if (live) Dc[(size_t)sub * N + n] = run;
    run = 1.f;
#pragma unroll
    for (int i = GLA_SUB - 1; i >= 0; --i) {
      if (i < own) K[at0 + i * step] = ks[(sub * GLA_SUB + i) * LA_LD + d] * run;
      run *= z[i];
    }
    __syncthreads();
    if (sub == 0 && live)
      Dc[(size_t)4 * N + n] = (tot[d] * tot[LA_BLK + d]) * (tot[2 * LA_BLK + d] * tot[3 * LA_BLK + d]);
    // pairs inside the sub-chunk: k_j times the decays after j, from token to token
    float4 pair[4];
#pragma unroll
    for (int a = 0; a < 4; ++a) pair[a] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < GLA_SUB; ++i) {
      const float4 q4 = *reinterpret_cast<const float4*>(qs + (sub * GLA_SUB + i) * LA_LD + 4 * sl);
      const float4 a4 = *reinterpret_cast<const float4*>(as + (sub * GLA_SUB + i) * LA_LD + 4 * sl);
      const float4 k4 = *reinterpret_cast<const float4*>(ks + (sub * GLA_SUB + i) * LA_LD + 4 * sl);
#pragma unroll
      for (int a = 0; a < 4; ++a) {
        const bool own = i == 4 * jq + a;
        pair[a].x = own ? k4.x : pair[a].x * a4.x;
        pair[a].y = own ? k4.y : pair[a].y * a4.y;
        pair[a].z = own ? k4.z : pair[a].z * a4.z;
        pair[a].w = own ? k4.w : pair[a].w * a4.w;
        p[a][i] = fmaf(q4.x, pair[a].x, p[a][i]);
        p[a][i] = fmaf(q4.y, pair[a].y, p[a][i]);
        p[a][i] = fmaf(q4.z, pair[a].z, p[a][i]);
        p[a][i] = fmaf(q4.w, pair[a].w, p[a][i]);
      }
    }
  }
  // sum over the sixteen lanes that share the key tokens: lane sl is left with query token sl
#pragma unroll
  for (int a = 0; a < 4; ++a) {
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) {
      const bool up = (sl & o) != 0;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (i >= o) break;
        const float send = up ? p[a][i] : p[a][i + o], keep = up ? p[a][i + o] : p[a][i];
        p[a][i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
      }
    }
    diag[(((size_t)tile * heads + h) * LA_C + sub * GLA_SUB + sl) * GLA_SUB + 4 * jq + a] = p[a][0];
  }
}

// A block takes NB x NB entries of a chunk's sum, a thread E x E of them (NB = 16 E).
template <typename T, int E>
__global__ void __launch_bounds__(256)
gla_chunk_kv_kernel(float* __restrict__ sums, GlaIn<T> in, const float* __restrict__ K, const float* __restrict__ D,
                    const int* __restrict__ q_tiles, const int* __restrict__ cu_tokens, int heads, int N, int M) {
  pdl_launch_dependents();
  constexpr int NB = 16 * E, LD = NB + 4, B = 4;
  extern __shared__ __align__(16) float sm[];
  float* Ks = sm;                              // [token][LD]
  float* Vs = sm + LA_C * LD;                  // [token][LD]
  float* after = Vs + LA_C * LD;               // [sub-chunk][NB]: the decays of the sub-chunks after it
  const int tile = blockIdx.x, h = blockIdx.y;
  const int vblocks = (M + NB - 1) / NB;
  const int n0 = (blockIdx.z / vblocks) * NB, m0 = (blockIdx.z % vblocks) * NB;
  int tok0 = 0;
  const int n_tok = la_tile_tokens(q_tiles, cu_tokens, tile, tok0);
  pdl_wait();
  if (n_tok == 0) return;
  if (threadIdx.x < NB) {
    const int n = n0 + threadIdx.x;
    const float* Dc = D + ((size_t)tile * heads + h) * 5 * N + (n < N ? n : 0);
    const float d1 = Dc[N], d2 = Dc[2 * (size_t)N], d3 = Dc[3 * (size_t)N];
    after[threadIdx.x] = d1 * (d2 * d3);
    after[NB + threadIdx.x] = d2 * d3;
    after[2 * NB + threadIdx.x] = d3;
    after[3 * NB + threadIdx.x] = 1.f;
  }
  __syncthreads();
  const bool vec_k = (N & 3) == 0;
  for (int i0 = threadIdx.x; i0 < n_tok * (NB / 4); i0 += 256 * B) {
    float k4[B][4], v4[B][4];
#pragma unroll
    for (int b = 0; b < B; ++b) {
      const int i = i0 + 256 * b, j = i / (NB / 4), d = (i - j * (NB / 4)) * 4;
      const int t = tok0 + (j < n_tok ? j : 0);
      gla_load4(K + ((size_t)t * heads + h) * N + n0 + d, N - n0 - d, vec_k, k4[b]);
      gla_load4(in.rows + (size_t)t * in.ld + in.v_off + (size_t)h * M + m0 + d, M - m0 - d, in.vec, v4[b]);
    }
#pragma unroll
    for (int b = 0; b < B; ++b) {
      const int i = i0 + 256 * b, j = i / (NB / 4), d = (i - j * (NB / 4)) * 4;
      if (j >= n_tok) continue;
      const float4 f = *reinterpret_cast<const float4*>(after + (j / GLA_SUB) * NB + d);
      *reinterpret_cast<float4*>(Ks + j * LD + d) = make_float4(k4[b][0] * f.x, k4[b][1] * f.y, k4[b][2] * f.z, k4[b][3] * f.w);
      *reinterpret_cast<float4*>(Vs + j * LD + d) = make_float4(v4[b][0], v4[b][1], v4[b][2], v4[b][3]);
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
// to the end of the request's tokens.  A thread W neighbouring entries of one row of S; a request's
// chunks in order.
template <int W>
__global__ void __launch_bounds__(256)
gla_states_kernel(float* __restrict__ sums, float* __restrict__ state, long state_stride, const float* __restrict__ D,
                  const int* __restrict__ cu_tokens, const int* __restrict__ slots, int heads, int N, int M) {
  pdl_launch_dependents();
  __shared__ int before[8];
  const int h = blockIdx.y, seq = blockIdx.z, NM = N * M;
  // chunks of the requests before this one
  int c = 0;
  for (int s = threadIdx.x; s < seq; s += 256) c += (cu_tokens[s + 1] - cu_tokens[s] + LA_C - 1) / LA_C;
  for (int w = 16; w > 0; w >>= 1) c += __shfl_xor_sync(0xffffffffu, c, w);
  if ((threadIdx.x & 31) == 0) before[threadIdx.x >> 5] = c;
  __syncthreads();
  int tile = 0;
  for (int w = 0; w < 8; ++w) tile += before[w];
  const int chunks = (cu_tokens[seq + 1] - cu_tokens[seq] + LA_C - 1) / LA_C;
  pdl_wait();
  const int e = (blockIdx.x * 256 + threadIdx.x) * W;
  if (e >= NM || chunks == 0) return;
  float* mine = state + (size_t)slots[seq] * state_stride + (size_t)h * NM + e;
  float s[W];
#pragma unroll
  for (int w = 0; w < W; ++w) s[w] = mine[w];
  const size_t step = (size_t)heads * NM, dstep = (size_t)heads * 5 * N;
  float* u = sums + ((size_t)tile * heads + h) * NM + e;
  const float* dec = D + (((size_t)tile * heads + h) * 5 + 4) * N + e / M;
  constexpr int AHEAD = 8;
  for (int k0 = 0; k0 < chunks; k0 += AHEAD) {
    float v[AHEAD][W], f[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
      if (k0 + k < chunks) {
        if constexpr (W == 4) la_load4(u + (size_t)(k0 + k) * step, v[k]);
        else v[k][0] = u[(size_t)(k0 + k) * step];
        f[k] = dec[(size_t)(k0 + k) * dstep];
      }
    }
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
      if (k0 + k < chunks) {
        float* dst = u + (size_t)(k0 + k) * step;
        if constexpr (W == 4) la_store4(dst, s);
        else *dst = s[0];
#pragma unroll
        for (int w = 0; w < W; ++w) s[w] = fmaf(f[k], s[w], v[k][w]);
      }
    }
  }
#pragma unroll
  for (int w = 0; w < W; ++w) mine[w] = s[w];
}

__device__ __forceinline__ void gla_copy16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

// VB: blocks of 64 columns of v a head has.  A thread owns the query tokens ty + 16 r (r is their
// sub-chunk) and, of the scores, the key tokens tx + 16 c; of the output, the columns 4 tx + e of
// every block.
template <typename T, int VB>
__global__ void __launch_bounds__(256)
gla_chunk_out_kernel(T* __restrict__ out, int out_ld, GlaIn<T> in, const float* __restrict__ Q,
                     const float* __restrict__ K, const float* __restrict__ D, const float* __restrict__ diag,
                     const float* __restrict__ states, const int* __restrict__ q_tiles,
                     const int* __restrict__ cu_tokens, int heads, int N, int M, const float* __restrict__ norm_weight,
                     float eps, float factor) {
  pdl_launch_dependents();
  constexpr int LDB = VB * LA_BLK + 4;
  extern __shared__ __align__(16) float sm[];
  float* Qs = sm;                              // [token][LA_LD]: 64 columns of Q, later the scores
  float* Ks = Qs + LA_C * LA_LD;               // [token][LA_LD]: 64 columns of K
  float* Bs = Ks + LA_C * LA_LD;               // 64 rows of S, later of v: [row][LDB]
  float* Ds = Bs + LA_BLK * LDB;               // [sub-chunk][64]
  const int tile = blockIdx.x, h = blockIdx.y;
  int tok0 = 0;
  const int n_tok = la_tile_tokens(q_tiles, cu_tokens, tile, tok0);
  pdl_wait();
  if (n_tok == 0) return;
  const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
  float p[4][4] = {};
  float acc[4][4 * VB] = {};
  const float* S = states + ((size_t)tile * heads + h) * N * M;
  const float* Dc = D + ((size_t)tile * heads + h) * 5 * N;
  const bool rows16 = (M & 3) == 0;            // rows of S begin at 16-byte boundaries
  const bool keys16 = (N & 3) == 0;            // ... of Q and K
  for (int n0 = 0; n0 < N; n0 += LA_BLK) {
    if (n0 > 0) __syncthreads();
    const int inner = min(LA_BLK, N - n0);
    for (int i = threadIdx.x; i < LA_C * (LA_BLK / 4); i += 256) {
      const int j = i / (LA_BLK / 4), d = (i - j * (LA_BLK / 4)) * 4;
      const size_t at = ((size_t)(tok0 + (j < n_tok ? j : 0)) * heads + h) * N + n0 + d;
      float* qd = Qs + j * LA_LD + d;
      float* kd = Ks + j * LA_LD + d;
      if (keys16 && j < n_tok && d < inner) {
        gla_copy16(qd, Q + at);
        gla_copy16(kd, K + at);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const bool ok = j < n_tok && d + e < inner;
          qd[e] = ok ? Q[at + e] : 0.f;
          kd[e] = ok ? K[at + e] : 0.f;
        }
      }
    }
    {
      const int s = threadIdx.x >> 6, d = threadIdx.x & 63;
      Ds[s * LA_BLK + d] = d < inner ? Dc[(size_t)s * N + n0 + d] : 0.f;
    }
    asm volatile("cp.async.commit_group;\n" ::);
    for (int i = threadIdx.x; i < LA_BLK * VB * (LA_BLK / 4); i += 256) {
      const int d = i / (VB * (LA_BLK / 4)), m = (i - d * (VB * (LA_BLK / 4))) * 4;
      float* dst = Bs + d * LDB + m;
      if (rows16 && d < inner && m < M) {
        gla_copy16(dst, S + (size_t)(n0 + d) * M + m);
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
    asm volatile("cp.async.wait_group 1;\n" ::);
    __syncthreads();
    const int steps = (inner + 3) & ~3;        // zeros beyond `inner`
    // scores of pairs in different sub-chunks (rows of sub-chunk r, keys of sub-chunks c < r)
#pragma unroll 2
    for (int d = 0; d < steps; d += 4) {
      float x[4][4], y[3][4], d1[4], d2[4];
#pragma unroll
      for (int r = 1; r < 4; ++r) {
        *reinterpret_cast<float4*>(x[r]) = *reinterpret_cast<const float4*>(Qs + (ty + 16 * r) * LA_LD + d);
        *reinterpret_cast<float4*>(y[r - 1]) = *reinterpret_cast<const float4*>(Ks + (tx + 16 * (r - 1)) * LA_LD + d);
      }
      *reinterpret_cast<float4*>(d1) = *reinterpret_cast<const float4*>(Ds + LA_BLK + d);
      *reinterpret_cast<float4*>(d2) = *reinterpret_cast<const float4*>(Ds + 2 * LA_BLK + d);
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        p[1][0] = fmaf(x[1][u], y[0][u], p[1][0]);
        p[2][1] = fmaf(x[2][u], y[1][u], p[2][1]);
        p[3][2] = fmaf(x[3][u], y[2][u], p[3][2]);
        const float y0 = y[0][u] * d1[u];
        p[2][0] = fmaf(x[2][u], y0, p[2][0]);
        p[3][1] = fmaf(x[3][u], y[1][u] * d2[u], p[3][1]);
        p[3][0] = fmaf(x[3][u], y0 * d2[u], p[3][0]);
      }
    }
    __syncthreads();
    // the state's share wants the decays from the chunk's start on
    for (int i = threadIdx.x; i < LA_C * (LA_BLK / 4); i += 256) {
      const int j = i / (LA_BLK / 4), d = (i - j * (LA_BLK / 4)) * 4;
      if (j < GLA_SUB) continue;
      float4 q4 = *reinterpret_cast<const float4*>(Qs + j * LA_LD + d);
      for (int s = 0; s < j / GLA_SUB; ++s) {
        const float4 f = *reinterpret_cast<const float4*>(Ds + s * LA_BLK + d);
        q4 = make_float4(q4.x * f.x, q4.y * f.y, q4.z * f.z, q4.w * f.w);
      }
      *reinterpret_cast<float4*>(Qs + j * LA_LD + d) = q4;
    }
    asm volatile("cp.async.wait_group 0;\n" ::);
    __syncthreads();
    la_rows_times<VB>(acc, Qs, Bs, ty, tx, steps);
  }
  __syncthreads();
  {
    const float* own = diag + ((size_t)tile * heads + h) * LA_C * GLA_SUB;
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
      for (int c = 0; c < 4; ++c)
        Qs[(ty + 16 * r) * LA_LD + tx + 16 * c] =
            c < r ? p[r][c] : c == r && tx <= ty ? own[(ty + 16 * r) * GLA_SUB + tx] : 0.f;
  }
  const int key_steps = (n_tok + 3) & ~3;
  {
    constexpr int B = 4, PER = VB * (LA_BLK / 4);
    for (int i0 = threadIdx.x; i0 < key_steps * PER; i0 += 256 * B) {
      float v[B][4];
#pragma unroll
      for (int b = 0; b < B; ++b) {
        const int i = i0 + 256 * b, j = i / PER, m = (i - j * PER) * 4;
        const int t = tok0 + (j < n_tok ? j : 0);
        gla_load4(in.rows + (size_t)t * in.ld + in.v_off + (size_t)h * M + m, j < n_tok ? M - m : 0, in.vec, v[b]);
      }
#pragma unroll
      for (int b = 0; b < B; ++b) {
        const int i = i0 + 256 * b, j = i / PER, m = (i - j * PER) * 4;
        if (j < key_steps) *reinterpret_cast<float4*>(Bs + j * LDB + m) = make_float4(v[b][0], v[b][1], v[b][2], v[b][3]);
      }
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
    float ss = 0.f;               // the sixteen threads of a row are neighbouring lanes
#pragma unroll
    for (int e = 0; e < 4 * VB; ++e) ss = fmaf(acc[r][e], acc[r][e], ss);
#pragma unroll
    for (int w = 8; w > 0; w >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
    if (j >= n_tok) continue;
    const int t = tok0 + j;
    const float rstd = factor * rsqrtf(ss / (float)M + eps);
#pragma unroll
    for (int vb = 0; vb < VB; ++vb) {
      const int m = vb * LA_BLK + 4 * tx;
      const T* g = in.rows + (size_t)t * in.ld + in.g_off + (size_t)h * M + m;
      T* dst = out + (size_t)t * out_ld + (size_t)h * M + m;
      float g4[4], y4[4];
      gla_load4(g, M - m, in.vec_gate, g4);
#pragma unroll
      for (int e = 0; e < 4; ++e)
        y4[e] = acc[r][4 * vb + e] * rstd * (m + e < M ? norm_weight[m + e] : 0.f) * la_gate(g4[e], 0);
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

template <typename T>
GlaIn<T> gla_in(const void* rows, int ld, int q_off, int k_off, int v_off, int g_off, int a_off, const void* w2,
                const float* bias, int R, float inv_tau, float q_scale, int N, int M, const void* out, int out_ld) {
  GlaIn<T> in;
  in.rows = (const T*)rows; in.ld = ld;
  in.q_off = q_off; in.k_off = k_off; in.v_off = v_off; in.g_off = g_off; in.a_off = a_off;
  in.w2 = (const T*)w2; in.bias = bias; in.R = R;
  in.inv_tau = inv_tau; in.q_scale = q_scale;
  in.vec = ((ld | v_off | M) & 3) == 0 && ((uintptr_t)rows & 15) == 0;
  in.vec_gate = ((ld | g_off | M | out_ld) & 3) == 0 && (((uintptr_t)rows | (uintptr_t)out) & 15) == 0;
  in.vec_w2 = (R & 3) == 0 && ((uintptr_t)w2 & 15) == 0;
  return in;
}

template <typename K>
bool gla_configure(K kernel, size_t smem, size_t& most) {
  if (smem <= 48 * 1024 || smem <= most) return true;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return false;
  most = smem;
  return true;
}

template <typename T, int E>
int gla_launch_kv(float* sums, const GlaIn<T>& in, const float* K, const float* D, const int* q_tiles, int n_tiles,
                  const int* cu_tokens, int heads, int N, int M, cudaStream_t stream) {
  constexpr int NB = 16 * E;
  constexpr size_t SMEM = (2 * LA_C * (NB + 4) + GLA_SUBS * NB) * sizeof(float);
  static size_t most = 0;
  if (!gla_configure(gla_chunk_kv_kernel<T, E>, SMEM, most)) return HB_LAUNCH_FAILED;
  hb_launch(gla_chunk_kv_kernel<T, E>, dim3(n_tiles, heads, ((N + NB - 1) / NB) * ((M + NB - 1) / NB)), dim3(256), SMEM,
            stream, sums, in, K, D, q_tiles, cu_tokens, heads, N, M);
  return hb_check_launch();
}

template <typename T, int VB>
int gla_launch_out(T* out, int out_ld, const GlaIn<T>& in, const float* Q, const float* K, const float* D,
                   const float* diag, const float* states, const int* q_tiles, int n_tiles, const int* cu_tokens,
                   int heads, int N, int M, const float* norm_weight, float eps, float factor, cudaStream_t stream) {
  constexpr size_t SMEM = (2 * LA_C * LA_LD + LA_BLK * (VB * LA_BLK + 4) + GLA_SUBS * LA_BLK) * sizeof(float);
  static size_t most = 0;
  if (!gla_configure(gla_chunk_out_kernel<T, VB>, SMEM, most)) return HB_LAUNCH_FAILED;
  hb_launch(gla_chunk_out_kernel<T, VB>, dim3(n_tiles, heads), dim3(256), SMEM, stream, out, out_ld, in, Q, K, D, diag,
            states, q_tiles, cu_tokens, heads, N, M, norm_weight, eps, factor);
  return hb_check_launch();
}

constexpr int GLA_MOST_RANK = 256;

}  // namespace

// rows [T, ld]: q, k (heads x N), v and the gate (heads x M), the low-rank columns (R) at the given
// columns.  w2 [heads * N, R] in the rows' type.  `o` null (M <= 128): norm and gate are applied and
// `out` (rows out_ld apart) is written; else o [T, heads, M] float32.
HB_EXPORT int hb_gla_scan(float* o, void* out, int out_ld, const void* rows, int ld, int q_off, int k_off, int v_off,
                          int g_off, int a_off, const void* w2, const float* bias, int R, float inv_tau, float q_scale,
                          float* state, long state_stride, const int* cu_tokens, const int* slots, int T, int S,
                          int heads, int N, int M, const float* norm_weight, float eps, float factor, int act_dt,
                          cudaStream_t stream) {
  if (T <= 0 || S <= 0) return HB_OK;
  if (N <= 0 || N > 256 || M <= 0 || heads <= 0 || R <= 0 || R > GLA_MOST_RANK || (o == nullptr && M > 128) ||
      w2 == nullptr || bias == nullptr || norm_weight == nullptr)
    return HB_BAD_ARGUMENT;
  const int vec = M <= 32 ? 1 : M <= 64 ? 2 : 4;
  const dim3 grid((M + 32 * vec - 1) / (32 * vec), heads, S);
  const int vec_state = M % vec == 0 && state_stride % vec == 0 && ((uintptr_t)state & (4 * vec - 1)) == 0;
#define HB_GLA_SCAN(TA, RW, V)                                                                                \
  hb_launch(gla_scan_kernel<TA, RW, V>, grid, dim3(32 * LA_PARTS), 0, stream, o, (TA*)out, out_ld,              \
            gla_in<TA>(rows, ld, q_off, k_off, v_off, g_off, a_off, w2, bias, R, inv_tau, q_scale, N, M, out, out_ld), \
            state, state_stride, cu_tokens, slots, heads, N, M, vec_state, norm_weight, eps, factor)
#define HB_GLA_SCAN_V(TA, V)                                                                                  \
  do {                                                                                                         \
    if (N <= 32) HB_GLA_SCAN(TA, 4, V);                                                                        \
    else if (N <= 64) HB_GLA_SCAN(TA, 8, V);                                                                   \
    else if (N <= 128) HB_GLA_SCAN(TA, 16, V);                                                                 \
    else HB_GLA_SCAN(TA, 32, V);                                                                               \
  } while (0)
  HB_DISPATCH_DTYPE(act_dt, TA,
    if (vec == 1) HB_GLA_SCAN_V(TA, 1);
    else if (vec == 2) HB_GLA_SCAN_V(TA, 2);
    else HB_GLA_SCAN_V(TA, 4));
#undef HB_GLA_SCAN_V
#undef HB_GLA_SCAN
  return hb_check_launch();
}

// Chunked.  Scratch, all float32 and 16-byte aligned: Q and K [T, heads, N], D [tiles, heads, 5, N],
// diag [tiles, heads, 64, 16], sums [tiles, heads, N, M].
HB_EXPORT int hb_gla_chunked(void* out, int out_ld, float* Q, float* K, float* D, float* diag, float* sums,
                             const void* rows, int ld, int q_off, int k_off, int v_off, int g_off, int a_off,
                             const void* w2, const float* bias, int R, float inv_tau, float q_scale, float* state,
                             long state_stride, const int* q_tiles, int n_tiles, const int* cu_tokens, const int* slots,
                             int S, int heads, int N, int M, const float* norm_weight, float eps, float factor,
                             int act_dt, cudaStream_t stream) {
  if (n_tiles <= 0 || S <= 0) return HB_OK;
  if (N <= 0 || N > 256 || M <= 0 || M > 256 || heads <= 0 || R <= 0 || R > GLA_MOST_RANK || w2 == nullptr ||
      bias == nullptr || norm_weight == nullptr ||
      (((uintptr_t)Q | (uintptr_t)K | (uintptr_t)D | (uintptr_t)diag | (uintptr_t)sums) & 15))
    return HB_BAD_ARGUMENT;
  HB_DISPATCH_DTYPE(act_dt, TA, {
    const GlaIn<TA> in = gla_in<TA>(rows, ld, q_off, k_off, v_off, g_off, a_off, w2, bias, R, inv_tau, q_scale, N, M,
                                    out, out_ld);
    const size_t smem = (3 * LA_C * LA_LD + GLA_SUBS * LA_BLK + LA_C * ((R + 3) & ~3)) * sizeof(float);
    static size_t most = 0;
    if (!gla_configure(gla_prepare_kernel<TA>, smem, most)) return HB_LAUNCH_FAILED;
    hb_launch(gla_prepare_kernel<TA>, dim3(n_tiles, heads), dim3(256), smem, stream, Q, K, D, diag, in, q_tiles,
              cu_tokens, heads, N);
    int st = hb_check_launch();
    if (st != HB_OK) return st;
    st = N > 64 || M > 64 ? gla_launch_kv<TA, 8>(sums, in, K, D, q_tiles, n_tiles, cu_tokens, heads, N, M, stream)
                          : gla_launch_kv<TA, 4>(sums, in, K, D, q_tiles, n_tiles, cu_tokens, heads, N, M, stream);
    if (st != HB_OK) return st;
    const int NM = N * M;
    if (M % 4 == 0)
      hb_launch(gla_states_kernel<4>, dim3((NM / 4 + 255) / 256, heads, S), dim3(256), 0, stream, sums, state,
                state_stride, D, cu_tokens, slots, heads, N, M);
    else
      hb_launch(gla_states_kernel<1>, dim3((NM + 255) / 256, heads, S), dim3(256), 0, stream, sums, state, state_stride,
                D, cu_tokens, slots, heads, N, M);
    const int vb = (M + LA_BLK - 1) / LA_BLK;
    if (vb == 1)
      st = gla_launch_out<TA, 1>((TA*)out, out_ld, in, Q, K, D, diag, sums, q_tiles, n_tiles, cu_tokens, heads, N, M, norm_weight, eps, factor, stream);
    else if (vb == 2)
      st = gla_launch_out<TA, 2>((TA*)out, out_ld, in, Q, K, D, diag, sums, q_tiles, n_tiles, cu_tokens, heads, N, M, norm_weight, eps, factor, stream);
    else
      st = gla_launch_out<TA, 4>((TA*)out, out_ld, in, Q, K, D, diag, sums, q_tiles, n_tiles, cu_tokens, heads, N, M, norm_weight, eps, factor, stream);
    return st;
  });
  return HB_OK;
}
