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

// A block a token; the blocks whose token ends no whole block of P tokens return at once.
template <typename T>
__global__ void __launch_bounds__(256)
pool_blocks_kernel(T* __restrict__ k_pooled, T* __restrict__ v_pooled, const int* __restrict__ pooled_table,
                   int pooled_stride, const T* __restrict__ k_pages, const T* __restrict__ v_pages,
                   const int* __restrict__ block_table, int bt_stride, const int* __restrict__ positions,
                   const int* __restrict__ seq_of_token, int nkv, int hd, int vd, int page_size, int pool) {
  pdl_launch_dependents();
  const int t = blockIdx.x;
  const int pos = positions[t], seq = seq_of_token[t];
  pdl_wait();
  if ((pos + 1) % pool != 0) return;
  const int block = pos / pool, first = block * pool;
  const int* table = block_table + (size_t)seq * bt_stride;
  const int page = pooled_table[(size_t)seq * pooled_stride + block / page_size];
  const int slot = block % page_size;
  const int per_head = hd + vd;
  const float inv = 1.f / (float)pool;
  for (int i = threadIdx.x; i < nkv * per_head; i += blockDim.x) {
    const int g = i / per_head, e = i - g * per_head;
    const bool is_k = e < hd;
    const int d = is_k ? e : e - hd, width = is_k ? hd : vd;
    const T* src = is_k ? k_pages : v_pages;
    float sum = 0.f;
    for (int j = 0; j < pool; ++j) {
      const int p = first + j;
      sum += to_float(src[(((size_t)table[p / page_size] * nkv + g) * page_size + p % page_size) * width + d]);
    }
    (is_k ? k_pooled : v_pooled)[(((size_t)page * nkv + g) * page_size + slot) * width + d] = from_float<T>(sum * inv);
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
  HB_DISPATCH_DTYPE(act_dt, TA,
    hb_launch(pool_blocks_kernel<TA>, dim3(T), dim3(256), 0, stream, (TA*)k_pooled, (TA*)v_pooled, pooled_table,
              pooled_stride, (const TA*)k_pages, (const TA*)v_pages, block_table, bt_stride, positions, seq_of_token,
              nkv, hd, vd, page_size, pool));
  return hb_check_launch();
}
