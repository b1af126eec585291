// What grouped-query window attention with pooled blocks does ahead of its scores
// (the scores themselves: attention_generic.cu and the tensor-core kernels).
//
//   conv_norm_rotate_write  q | k | v columns of a fused projection: a short causal convolution
//       over time per channel (zeros before the request's start, the inputs before the step's
//       first token from the request's slot), an RMS norm per q and k head with a weight, a
//       rotation of the first `rot` values of q and k (value i paired with value i + rot / 2);
//       q goes to rows of its own, k and v to the request's pages.  Between the projection and
//       the stores everything stays in float32 registers.
//   pool_blocks  for every token that ends a whole block of P tokens: the means of the block's
//       keys and values as the pages hold them, as one row of the pooled pages.
#include "common.cuh"
#include "causal_conv.cuh"

namespace {

constexpr int CW_WARPS = 4;
constexpr int CW_MAX = 256;        // values a head

template <typename T>
struct CwArgs {
  T* q_out;                 // [T, nh * hd]
  T* k_pages;               // null: no cache write
  T* v_pages;
  const T* rows;            // [T, ld], q from column 0
  int ld;
  const float* conv;        // [nh hd + nkv hd + nkv vd, taps] or null
  float* state;             // a slot's inputs: [channels, taps - 1], oldest first
  long state_stride;
  int taps;
  const float* wq;
  const float* wk;
  float eps;
  const float* cos;         // [T, rot / 2]
  const float* sin;
  int rot;
  const int* positions;
  const int* seq_of_token;
  const int* cu_tokens;
  const int* slots;
  const int* block_table;
  int bt_stride;
  int n_tokens, nh, nkv, hd, vd, page_size;
  int single;               // every request has one token in the step: the slot's inputs move on here
};

// A warp a (token, head).
template <typename T>
__global__ void __launch_bounds__(CW_WARPS * 32)
conv_norm_rotate_write_kernel(CwArgs<T> a) {
  pdl_launch_dependents();
  __shared__ float head_row[CW_WARPS][CW_MAX];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int per_token = a.nh + 2 * a.nkv;
  const long item = (long)blockIdx.x * CW_WARPS + warp;
  pdl_wait();
  if (item >= (long)a.n_tokens * per_token) return;
  const int t = (int)(item / per_token), h = (int)(item - (long)t * per_token);
  const bool is_v = h >= a.nh + a.nkv, is_q = h < a.nh;
  const int n = is_v ? a.vd : a.hd;
  const int c0 = is_v ? (a.nh + a.nkv) * a.hd + (h - a.nh - a.nkv) * a.vd : h * a.hd;
  const int seq = a.seq_of_token[t], pos = a.positions[t];
  const int local = t - a.cu_tokens[seq];
  const T* row = a.rows + (size_t)t * a.ld + c0;
  float* x = head_row[warp];
  const int keep = a.taps - 1;
  float ss = 0.f;
  for (int d = lane; d < n; d += 32) {
    float v = to_float(row[d]);
    if (a.conv != nullptr) {
      const float* w = a.conv + (size_t)(c0 + d) * a.taps;
      float* st = a.state + (size_t)a.slots[seq] * a.state_stride + (size_t)(c0 + d) * keep;
      const float now = v;
      float acc = 0.f;
      for (int j = 0; j < keep; ++j) {
        const int src = local - keep + j;
        const float u = src >= 0 ? to_float(row[d - (long)(keep - j) * a.ld]) : st[keep + src];
        acc = fmaf(w[j], u, acc);
      }
      v = fmaf(w[keep], now, acc);
      if (a.single && keep > 0) {
        for (int j = 0; j + 1 < keep; ++j) st[j] = st[j + 1];
        st[keep - 1] = now;
      }
    }
    x[d] = v;
    ss = fmaf(v, v, ss);
  }
  size_t page_row = 0;
  if (!is_q && a.k_pages != nullptr) {
    const int page = a.block_table[(size_t)seq * a.bt_stride + pos / a.page_size];
    const int g = is_v ? h - a.nh - a.nkv : h - a.nh;
    page_row = ((size_t)page * a.nkv + g) * a.page_size + pos % a.page_size;
  }
  if (is_v) {
    if (a.v_pages == nullptr) return;
    for (int d = lane; d < n; d += 32) a.v_pages[page_row * a.vd + d] = from_float<T>(x[d]);
    return;
  }
  const float rstd = rsqrtf(warp_sum(ss) / (float)n + a.eps);
  const float* w = is_q ? a.wq : a.wk;
  if (!is_q && a.k_pages == nullptr) return;
  T* dst = is_q ? a.q_out + ((size_t)t * a.nh + h) * a.hd : a.k_pages + page_row * a.hd;
  __syncwarp();
  const int half = a.rot / 2;
  for (int d = lane; d < n; d += 32) {
    float v = x[d] * rstd * w[d];
    if (d < a.rot) {
      const int p = d < half ? d : d - half, other = d < half ? d + half : d - half;
      const float c = a.cos[(size_t)t * half + p], s = a.sin[(size_t)t * half + p];
      const float o = x[other] * rstd * w[other];
      v = d < half ? v * c - o * s : v * c + o * s;
    }
    dst[d] = from_float<T>(v);
  }
}

__device__ __forceinline__ void cw_load8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const uint32_t in[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&in[e]));
    f[2 * e] = v.x;
    f[2 * e + 1] = v.y;
  }
}
__device__ __forceinline__ void cw_store8(__nv_bfloat16* p, const float (&f)[8]) {
  uint32_t w[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(f[2 * e], f[2 * e + 1]);
    w[e] = *reinterpret_cast<const uint32_t*>(&v);
  }
  *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
}

// The same for bfloat16 in 16-byte pieces: a thread takes eight neighbouring channels of TOK
// consecutive tokens (their shared inputs and the channels' weights are read once), a group of
// GROUP lanes a q or k head (norm and rotation inside the group: rot / 2 is a multiple of 8, or
// there is no rotation); the blocks with blockIdx.y == 1 take the value heads.  Each channel's
// convolution is summed in the order of the kernel above.
template <int GROUP, int TAPS, int TOK>
__global__ void __launch_bounds__(128)
conv_norm_rotate_write_vec_kernel(CwArgs<__nv_bfloat16> a) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int HD = GROUP * 8, KEEP = TAPS - 1, ROWS = TOK + KEEP;
  const bool values = blockIdx.y == 1;
  const int per_group = values ? a.nkv * (a.vd >> 3) : (a.nh + a.nkv) * GROUP;
  const long tid = (long)blockIdx.x * blockDim.x + threadIdx.x;
  const long groups = (a.n_tokens + TOK - 1) / TOK;
  const bool live = tid < groups * per_group;      // whole groups of GROUP lanes live or die together
  const int tg = live ? (int)(tid / per_group) : 0, piece = live ? (int)(tid - (long)tg * per_group) : 0;
  const int t0 = tg * TOK;
  const int c = (values ? (a.nh + a.nkv) * HD : 0) + piece * 8;       // first channel of the thread
  const int head = values ? piece / (a.vd >> 3) : piece / GROUP;
  const int d0 = values ? (piece - head * (a.vd >> 3)) * 8 : (piece % GROUP) * 8;
  if (values && (!live || a.v_pages == nullptr)) {
    if (!live || KEEP == 0 || !a.single) return;
  }
  float w[8 * TAPS];
  if (a.conv != nullptr) {
    // eight channels' weights are 8 x TAPS consecutive floats from a 32-byte boundary
#pragma unroll
    for (int i = 0; i < 2 * TAPS; ++i) {
      const float4 q = *reinterpret_cast<const float4*>(a.conv + (size_t)c * TAPS + 4 * i);
      w[4 * i] = q.x; w[4 * i + 1] = q.y; w[4 * i + 2] = q.z; w[4 * i + 3] = q.w;
    }
  }
  float x[ROWS][8];
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const int row = t0 - KEEP + r;
    if (live && row >= 0 && row < a.n_tokens) cw_load8(a.rows + (size_t)row * a.ld + c, x[r]);
    else {
#pragma unroll
      for (int e = 0; e < 8; ++e) x[r][e] = 0.f;
    }
  }
#pragma unroll
  for (int u = 0; u < TOK; ++u) {
    const int t = t0 + u;
    const bool on = live && t < a.n_tokens;
    const int seq = on ? a.seq_of_token[t] : 0;
    const int pos = on ? a.positions[t] : 0;
    float y[8];
    if (a.conv == nullptr) {
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = x[u + KEEP][e];
    } else {
      const int local = on ? t - a.cu_tokens[seq] : KEEP;
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = 0.f;
      if (local >= KEEP) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j)
#pragma unroll
          for (int e = 0; e < 8; ++e) y[e] = fmaf(w[e * TAPS + j], x[u + j][e], y[e]);
      } else {
        // the request's first tokens of this step: the inputs before them are in its slot
        float* st = a.state + (size_t)a.slots[seq] * a.state_stride + (size_t)c * KEEP;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
          const int src = local - KEEP + j;
#pragma unroll
          for (int e = 0; e < 8; ++e)
            y[e] = fmaf(w[e * TAPS + j], src >= 0 ? x[u + j][e] : st[(size_t)e * KEEP + KEEP + src], y[e]);
        }
        if (a.single) {
#pragma unroll
          for (int e = 0; e < 8; ++e) {
#pragma unroll
            for (int j = 0; j + 1 < KEEP; ++j) st[(size_t)e * KEEP + j] = st[(size_t)e * KEEP + j + 1];
            st[(size_t)e * KEEP + KEEP - 1] = x[u + KEEP][e];
          }
        }
      }
    }
    size_t page_row = 0;
    const int g = values ? head : head - a.nh;
    if (on && (values || head >= a.nh) && a.k_pages != nullptr) {
      const int page = a.block_table[(size_t)seq * a.bt_stride + pos / a.page_size];
      page_row = ((size_t)page * a.nkv + g) * a.page_size + pos % a.page_size;
    }
    if (values) {
      if (on && a.v_pages != nullptr) cw_store8(a.v_pages + page_row * a.vd + d0, y);
      continue;
    }
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(y[e], y[e], ss);
#pragma unroll
    for (int o = GROUP / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float rstd = rsqrtf(ss / (float)HD + a.eps);
    const bool is_q = head < a.nh;
    const float* nw = (is_q ? a.wq : a.wk) + d0;
#pragma unroll
    for (int e = 0; e < 8; ++e) y[e] *= rstd * nw[e];
    if (a.rot > 0) {
      const int half = a.rot / 2, hp = half / 8;          // pieces of 8 in half a rotation
      const int me = d0 / 8;
      const bool lower = me < hp, turned = me < 2 * hp;
      const int other = lower ? me + hp : me - hp;
      const int src = turned ? (threadIdx.x & 31 & ~(GROUP - 1)) + other : (threadIdx.x & 31);
      float z[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) z[e] = __shfl_sync(0xffffffffu, y[e], src);
      if (on && turned) {
        const size_t at = (size_t)t * half + (lower ? d0 : d0 - half);
        const float sg = lower ? -1.f : 1.f;
        float cs[8], sn[8];                               // half is a multiple of 8
#pragma unroll
        for (int e = 0; e < 8; e += 4) {
          *reinterpret_cast<float4*>(cs + e) = *reinterpret_cast<const float4*>(a.cos + at + e);
          *reinterpret_cast<float4*>(sn + e) = *reinterpret_cast<const float4*>(a.sin + at + e);
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] = y[e] * cs[e] + sg * z[e] * sn[e];
      }
    }
    if (on) {
      if (is_q) cw_store8(a.q_out + ((size_t)t * a.nh + head) * HD + d0, y);
      else if (a.k_pages != nullptr) cw_store8(a.k_pages + page_row * HD + d0, y);
    }
  }
}

template <int GROUP, int TAPS>
void cw_launch_vec(const CwArgs<__nv_bfloat16>& a, cudaStream_t stream) {
  const int tok = a.n_tokens >= 256 ? 4 : 1;
  const long groups = (a.n_tokens + tok - 1) / tok;
  const long qk = groups * (a.nh + a.nkv) * GROUP, vals = groups * a.nkv * (a.vd / 8);
  const dim3 grid((unsigned)(((qk > vals ? qk : vals) + 127) / 128), 2);
  if (tok == 4) hb_launch(conv_norm_rotate_write_vec_kernel<GROUP, TAPS, 4>, grid, dim3(128), 0, stream, a);
  else hb_launch(conv_norm_rotate_write_vec_kernel<GROUP, TAPS, 1>, grid, dim3(128), 0, stream, a);
}

template <int GROUP>
void cw_launch_group(const CwArgs<__nv_bfloat16>& a, cudaStream_t stream) {
  if (a.taps == 1) cw_launch_vec<GROUP, 1>(a, stream);
  else if (a.taps == 2) cw_launch_vec<GROUP, 2>(a, stream);
  else if (a.taps == 3) cw_launch_vec<GROUP, 3>(a, stream);
  else cw_launch_vec<GROUP, 4>(a, stream);
}

inline bool cw_vec_fits(const CwArgs<float>&) { return false; }
inline bool cw_vec_fits(const CwArgs<__nv_bfloat16>& a) {
  const int group = a.hd / 8;
  return a.hd % 8 == 0 && a.vd % 8 == 0 && a.ld % 8 == 0 && (group == 4 || group == 8 || group == 16 || group == 32) &&
         a.taps <= 4 && (a.rot / 2) % 8 == 0 &&
         (((uintptr_t)a.rows | (uintptr_t)a.q_out | (uintptr_t)a.k_pages | (uintptr_t)a.v_pages | (uintptr_t)a.conv |
           (uintptr_t)a.cos | (uintptr_t)a.sin) & 15) == 0;
}
inline void cw_launch(const CwArgs<float>&, cudaStream_t) {}
inline void cw_launch(const CwArgs<__nv_bfloat16>& a, cudaStream_t stream) {
  const int group = a.hd / 8;
  if (group == 4) cw_launch_group<4>(a, stream);
  else if (group == 8) cw_launch_group<8>(a, stream);
  else if (group == 16) cw_launch_group<16>(a, stream);
  else cw_launch_group<32>(a, stream);
}

// A block a token; the blocks whose token ends no whole block of P tokens return at once.  A
// thread W neighbouring values, summed in the order of the tokens.
constexpr int POOL_ROWS = 1024;    // tokens a block whose places are looked up once

template <typename T, int W>
__global__ void __launch_bounds__(256)
pool_blocks_kernel(T* __restrict__ k_pooled, T* __restrict__ v_pooled, const int* __restrict__ pooled_table,
                   int pooled_stride, const T* __restrict__ k_pages, const T* __restrict__ v_pages,
                   const int* __restrict__ block_table, int bt_stride, const int* __restrict__ positions,
                   const int* __restrict__ seq_of_token, int nkv, int hd, int vd, int page_size, int pool) {
  pdl_launch_dependents();
  __shared__ int rows[POOL_ROWS];
  const int t = blockIdx.x;
  const int pos = positions[t], seq = seq_of_token[t];
  pdl_wait();
  if ((pos + 1) % pool != 0) return;
  const int block = pos / pool, first = block * pool;
  const int* table = block_table + (size_t)seq * bt_stride;
  auto row_of = [&](int p) { return table[p / page_size] * nkv * page_size + p % page_size; };
  for (int j = threadIdx.x; j < min(pool, POOL_ROWS); j += blockDim.x) rows[j] = row_of(first + j);
  __syncthreads();
  const int page = pooled_table[(size_t)seq * pooled_stride + block / page_size];
  const int slot = block % page_size;
  const float inv = 1.f / (float)pool;
  const int per_head = (hd + vd) / W;
  for (int i = threadIdx.x; i < nkv * per_head; i += blockDim.x) {
    const int g = i / per_head, e = (i - g * per_head) * W;
    const bool is_k = e < hd;
    const int d = is_k ? e : e - hd, width = is_k ? hd : vd;
    const T* src = (is_k ? k_pages : v_pages) + (size_t)g * page_size * width + d;
    float sum[W];
#pragma unroll
    for (int w = 0; w < W; ++w) sum[w] = 0.f;
#pragma unroll 8
    for (int j = 0; j < pool; ++j) {
      const T* at = src + (size_t)(j < POOL_ROWS ? rows[j] : row_of(first + j)) * width;
      if constexpr (W == 8) {
        float v[8];
        cw_load8(at, v);
#pragma unroll
        for (int w = 0; w < W; ++w) sum[w] += v[w];
      } else {
        sum[0] += to_float(at[0]);
      }
    }
#pragma unroll
    for (int w = 0; w < W; ++w) sum[w] *= inv;
    T* dst = (is_k ? k_pooled : v_pooled) + (((size_t)page * nkv + g) * page_size + slot) * width + d;
    if constexpr (W == 8) cw_store8(dst, sum);
    else dst[0] = from_float<T>(sum[0]);
  }
}

}  // namespace

HB_EXPORT int hb_conv_norm_rotate_write(void* q_out, void* k_pages, void* v_pages, const void* rows, int ld,
                                        const float* conv, float* state, long state_stride, int taps,
                                        const float* wq, const float* wk, float eps, const float* cos_tab,
                                        const float* sin_tab, int rot, const int* positions,
                                        const int* seq_of_token, const int* cu_tokens, const int* slots,
                                        const int* block_table, int bt_stride, int T, int S, int nh, int nkv, int hd,
                                        int vd, int page_size, int single, int act_dt, cudaStream_t stream) {
  if (T <= 0) return HB_OK;
  const int channels = (nh + nkv) * hd + nkv * vd;
  if (nh <= 0 || nkv <= 0 || hd <= 0 || hd > CW_MAX || vd <= 0 || vd > CW_MAX || page_size <= 0 || rot < 0 ||
      rot % 2 || rot > hd || channels > ld || (conv != nullptr && taps < 1) ||
      (conv != nullptr && taps > 1 && state == nullptr) || (k_pages == nullptr) != (v_pages == nullptr) ||
      (rot > 0 && (!cos_tab || !sin_tab)))
    return HB_BAD_ARGUMENT;
  const long items = (long)T * (nh + 2 * nkv);
  HB_DISPATCH_DTYPE(act_dt, TA, {
    const CwArgs<TA> a = {(TA*)q_out, (TA*)k_pages, (TA*)v_pages, (const TA*)rows, ld, conv, state, state_stride,
                          conv ? taps : 1, wq, wk, eps, cos_tab, sin_tab, rot, positions, seq_of_token, cu_tokens,
                          slots, block_table, bt_stride, T, nh, nkv, hd, vd, page_size, single};
    if (cw_vec_fits(a))
      cw_launch(a, stream);
    else
      hb_launch(conv_norm_rotate_write_kernel<TA>, dim3((unsigned)((items + CW_WARPS - 1) / CW_WARPS)),
                dim3(CW_WARPS * 32), 0, stream, a);
    if (conv != nullptr && taps > 1 && !single) {
      size_t blocks = ((size_t)S * channels + 255) / 256;
      if (blocks > 148 * 16) blocks = 148 * 16;
      hb_launch(causal_conv_state_kernel<TA>, dim3((unsigned)blocks), dim3(256), 0, stream, state, state_stride,
                (const TA*)rows, ld, cu_tokens, slots, S, channels, taps);
    }
  });
  return hb_check_launch();
}

HB_EXPORT int hb_pool_blocks(void* k_pooled, void* v_pooled, const int* pooled_table, int pooled_stride,
                             const void* k_pages, const void* v_pages, const int* block_table, int bt_stride,
                             const int* positions, const int* seq_of_token, int T, int nkv, int hd, int vd,
                             int page_size, int pool, int act_dt, cudaStream_t stream) {
  if (T <= 0) return HB_OK;
  if (nkv <= 0 || hd <= 0 || vd <= 0 || page_size <= 0 || pool <= 0) return HB_BAD_ARGUMENT;
  const bool vec = act_dt == HB_BF16 && hd % 8 == 0 && vd % 8 == 0 &&
                   (((uintptr_t)k_pooled | (uintptr_t)v_pooled | (uintptr_t)k_pages | (uintptr_t)v_pages) & 15) == 0;
  if (vec) {
    using B = __nv_bfloat16;
    hb_launch(pool_blocks_kernel<B, 8>, dim3(T), dim3(128), 0, stream, (B*)k_pooled, (B*)v_pooled, pooled_table,
              pooled_stride, (const B*)k_pages, (const B*)v_pages, block_table, bt_stride, positions, seq_of_token, nkv,
              hd, vd, page_size, pool);
    return hb_check_launch();
  }
  HB_DISPATCH_DTYPE(act_dt, TA,
    hb_launch(pool_blocks_kernel<TA, 1>, dim3(T), dim3(256), 0, stream, (TA*)k_pooled, (TA*)v_pooled, pooled_table,
              pooled_stride, (const TA*)k_pages, (const TA*)v_pages, block_table, bt_stride, positions, seq_of_token,
              nkv, hd, vd, page_size, pool));
  return hb_check_launch();
}
