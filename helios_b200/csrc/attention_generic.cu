// Attention over the paged cache for any batch of tokens: one warp per
// (token, query head).  It serves the float32 path and every size the tiled
// bfloat16 kernels do not take.  A token at position p sees the keys at
// positions lo..p of its own request, lo = max(0, p - window + 1) with a
// window and 0 without, wherever the pages lie
// (python/helios/exec/paged_attn.py:264-295, 368-408; GQA mapping :248-261).
//
// Options, each off by default: values of another size than the keys (`vd`); a bias on the
// score that grows with the distance, score - slopes[h] * (p - j); a bias looked up by the
// distance, score + bias_table[min(p - j, bias_rows - 1), h]; first tokens that a window
// keeps (`keep_first`: j visible if j <= p and (p - j < window or j < keep_first)); a sink in
// the softmax, a key without a value whose score is 0 or sink_values[h], so that the weights
// are exp(s_j) / (exp(sink) + sum exp(s_j)); a gate per (token, head), the head's output times
// sigmoid(gate[t, h]), or per output value (`gate_wide`: gate[t, h * vd + d]); means of whole blocks
// of `pool` tokens behind the window (`pooled`: a key and a value a block in pages of their own,
// block b seen if (b + 1) * pool <= p - window + 1); a constant `factor` on the output.
//
// Scores, softmax and the weighted sum are float32.  The keys are walked in
// runs of 32 from `lo`, so the order of every sum depends on the token's
// position alone: not on how the request was cut into steps, nor on the rest of
// the batch.
#include "common.cuh"

// Keys and values that stand for whole blocks of tokens; all null / 0: none.
template <typename T>
struct PooledPages {
  const T* k;             // [page, kv head, slot, hd]
  const T* v;             // [page, kv head, slot, vd]
  const int* table;       // [requests, table_stride]
  int table_stride;
  int pool;
};

constexpr int ATTN_WARPS = 4;
constexpr int ATTN_MAX_HD = 256;

template <typename T>
__global__ void attention_generic_kernel(
    T* __restrict__ out, const T* __restrict__ q, int q_stride,
    const T* __restrict__ k_pages, const T* __restrict__ v_pages,
    const int* __restrict__ block_table, int bt_stride, const int* __restrict__ seq_of_token,
    const int* __restrict__ positions, int n_rows, int nh, int nkv, int hd, int vd, int page_size,
    int window, float scale, const float* __restrict__ slopes, int sink,
    const T* __restrict__ gate, int gate_stride, const float* __restrict__ bias_table, int bias_rows,
    const float* __restrict__ sink_values, int keep_first, int gate_wide, PooledPages<T> pooled,
    int out_stride, float factor) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float q_smem[ATTN_WARPS][ATTN_MAX_HD];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = blockIdx.x * ATTN_WARPS + warp;
  if (row >= n_rows) return;
  const int t = row / nh, h = row - t * nh;
  const int kvh = h / (nh / nkv);
  const int pos = positions[t];
  const int* token_table = block_table + (size_t)seq_of_token[t] * bt_stride;
  const int lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;

  float* qs = q_smem[warp];
  const T* qrow = q + (size_t)t * q_stride + (size_t)h * hd;
  for (int d = lane; d < hd; d += 32) qs[d] = to_float(qrow[d]);
  __syncwarp();

  constexpr int ND = ATTN_MAX_HD / 32;
  float acc[ND];
#pragma unroll
  for (int i = 0; i < ND; ++i) acc[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  const float slope = slopes ? slopes[h] : 0.f;

  // three stretches of keys: the means of the blocks behind the window, the first tokens a
  // window keeps (those it has passed), then the window itself; each in runs of 32 from its own
  // first key
  for (int stretch = pooled.pool > 0 ? -1 : 0; stretch < 2; ++stretch) {
    const int first = stretch <= 0 ? 0 : lo;
    const int last = stretch < 0 ? lo / pooled.pool - 1 : stretch == 0 ? min(keep_first, lo) - 1 : pos;
    const int* table = stretch < 0 ? pooled.table + (size_t)seq_of_token[t] * pooled.table_stride : token_table;
    const T* kp = stretch < 0 ? pooled.k : k_pages;
    const T* vp = stretch < 0 ? pooled.v : v_pages;
    for (int base = first; base <= last; base += 32) {
      const int key = base + lane;
      const bool valid = key <= last;
      int page = 0;
      float score = -INFINITY;
      if (valid) {
        page = table[key / page_size];
        const T* kr = kp + (((size_t)page * nkv + kvh) * page_size + key % page_size) * hd;
        float dot = 0.f;
        for (int d = 0; d < hd; ++d) dot = fmaf(qs[d], to_float(kr[d]), dot);
        score = dot * scale - slope * (float)(pos - key);
        if (bias_table) score += bias_table[(size_t)min(pos - key, bias_rows - 1) * nh + h];
      }
      const float m_new = fmaxf(m, warp_max(score));
      const float p = valid ? expf(score - m_new) : 0.f;
      const float corr = (m == -INFINITY) ? 0.f : expf(m - m_new);
      l = l * corr + warp_sum(p);
      m = m_new;
#pragma unroll
      for (int i = 0; i < ND; ++i) acc[i] *= corr;
      const int n_valid = min(32, last - base + 1);
      for (int j = 0; j < n_valid; ++j) {
        const float pj = __shfl_sync(0xffffffffu, p, j);
        const int pagej = __shfl_sync(0xffffffffu, page, j);
        const T* vr = vp + (((size_t)pagej * nkv + kvh) * page_size + (base + j) % page_size) * vd;
#pragma unroll
        for (int i = 0; i < ND; ++i) {
          const int d = lane + 32 * i;
          if (d < vd) acc[i] = fmaf(pj, to_float(vr[d]), acc[i]);
        }
      }
    }
  }
  if (sink) {                       // a key without a value: it adds exp(s - m) to the sum only (s = 0 unless given)
    const float sv = sink_values ? sink_values[h] : 0.f;
    const float m_new = fmaxf(m, sv);
    const float corr = expf(m - m_new);
    l = l * corr + expf(sv - m_new);
#pragma unroll
    for (int i = 0; i < ND; ++i) acc[i] *= corr;
  }
  float inv = factor / l;
  if (gate && !gate_wide) inv /= 1.f + expf(-to_float(gate[(size_t)t * gate_stride + h]));
  T* orow = out + (size_t)t * out_stride + (size_t)h * vd;
#pragma unroll
  for (int i = 0; i < ND; ++i) {
    const int d = lane + 32 * i;
    if (d < vd) {
      float y = acc[i] * inv;
      if (gate && gate_wide) y /= 1.f + expf(-to_float(gate[(size_t)t * gate_stride + (size_t)h * vd + d]));
      orow[d] = from_float<T>(y);
    }
  }
}

HB_EXPORT int hb_attention_generic(void* out, const void* q, int q_stride, const void* k_pages,
                                   const void* v_pages, const int* block_table, int bt_stride,
                                   const int* seq_of_token, const int* positions, int T, int nh,
                                   int nkv, int hd, int vd, int page_size, int window, float scale,
                                   const float* slopes, int sink, const void* gate,
                                   int gate_stride, const float* bias_table, int bias_rows,
                                   const float* sink_values, int keep_first, int gate_wide,
                                   const void* pooled_k, const void* pooled_v, const int* pooled_table,
                                   int pooled_table_stride, int pool, int out_stride, float factor, int act_dt,
                                   cudaStream_t stream) {
  if (T <= 0) return HB_OK;
  if (hd <= 0 || hd > ATTN_MAX_HD || vd <= 0 || vd > ATTN_MAX_HD || nkv <= 0 || nh % nkv != 0 ||
      page_size <= 0 || keep_first < 0 || pool < 0 || out_stride < nh * vd ||
      (pool > 0 && (window <= 0 || !pooled_k || !pooled_v || !pooled_table)) || (bias_table != nullptr && bias_rows <= 0))
    return HB_BAD_ARGUMENT;
  const int n_rows = T * nh;
  const int blocks = (n_rows + ATTN_WARPS - 1) / ATTN_WARPS;
  HB_DISPATCH_DTYPE(act_dt, TA,
    hb_launch(attention_generic_kernel<TA>, dim3(blocks), dim3(ATTN_WARPS * 32), 0, stream, 
        (TA*)out, (const TA*)q, q_stride, (const TA*)k_pages, (const TA*)v_pages, block_table,
        bt_stride, seq_of_token, positions, n_rows, nh, nkv, hd, vd, page_size, window, scale,
        slopes, sink, (const TA*)gate, gate_stride, bias_table, bias_rows, sink_values, keep_first,
        gate_wide,
        PooledPages<TA>{(const TA*)pooled_k, (const TA*)pooled_v, pooled_table, pooled_table_stride, pool},
        out_stride, factor));
  return hb_check_launch();
}
