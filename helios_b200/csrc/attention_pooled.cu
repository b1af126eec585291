// Decode attention with keys and values of sizes of their own up to 256 (attention_decode.cuh with
// POOLED), compiled for 64, 128 and 256 each: over a window's tokens and the means of whole blocks
// behind it, under one softmax, or over all tokens or a window's without such blocks; with a sink, a
// gate, and the q/k norm and cache write of the step's own tokens on the way in.
#include "attention_decode.cuh"

namespace {

constexpr int POOLED_WARPS = 4;

template <typename F>
int pooled_dispatch(int hd, int vd, F f) {
  auto values = [&](auto H) {
    constexpr int HD = decltype(H)::value;
    if (vd <= 64) return f(std::integral_constant<int, HD>(), std::integral_constant<int, 64>());
    if (vd <= 128) return f(std::integral_constant<int, HD>(), std::integral_constant<int, 128>());
    return f(std::integral_constant<int, HD>(), std::integral_constant<int, 256>());
  };
  if (hd <= 64) return values(std::integral_constant<int, 64>());
  if (hd <= 128) return values(std::integral_constant<int, 128>());
  if (hd <= 192) return values(std::integral_constant<int, 192>());
  return values(std::integral_constant<int, 256>());
}

bool pooled_sizes_ok(int hd, int vd) {
  return hd > 0 && hd <= 256 && hd % 8 == 0 && vd > 0 && vd <= 256 && vd % 8 == 0;
}

}  // namespace

// S requests, one token each (token i belongs to request i), q [S, nh * hd].  The step's keys and
// values are in the pages, and so is every block's row that ends before the window.  With
// `write_cache` the rows of q hold k [nkv * hd] and v [nkv * vd] behind the queries, and the kernel
// stores them first; wq / wk float [hd]: q (and such a k) still lacks its RMS norm with that weight.  part_o float
// [S, nh, n_splits, vd] and part_ml float [S, nh, n_splits, 2], or both null with n_splits of 1 or
// 2..8 slices that run as one thread-block cluster.
HB_EXPORT int hb_attention_pooled_decode(void* out, int out_stride, float factor, float* part_o, float* part_ml,
                                         const void* q, int q_stride, const void* k_pages, const void* v_pages,
                                         const int* block_table, int bt_stride, const void* pooled_k,
                                         const void* pooled_v, const int* pooled_table, int pooled_stride, int pool,
                                         const int* positions, int S, int nh, int nkv, int hd, int vd, int page_size,
                                         int window, float scale, int n_splits, int sink, const float* sink_values,
                                         const void* gate, int gate_stride, int gate_wide, int write_cache,
                                         const float* wq, const float* wk, float eps, cudaStream_t stream) {
  if (S <= 0) return HB_OK;
  if (!pooled_sizes_ok(hd, vd) || nkv <= 0 || nh % nkv != 0 || nh / nkv > 16 || page_size <= 0 || n_splits < 1 ||
      window < 0 || pool < 0 || (pool > 0 && window <= 0) || out_stride < nh * vd || (part_o == nullptr) != (part_ml == nullptr) ||
      (part_o == nullptr && n_splits > 8) || (pool > 0 && (!pooled_k || !pooled_v || !pooled_table)) ||
      (((uintptr_t)k_pages | (uintptr_t)v_pages | (uintptr_t)pooled_k | (uintptr_t)pooled_v) & 15) ||
      ((uintptr_t)q & 3) || (q_stride & 1) || (((uintptr_t)wq | (uintptr_t)wk) & 7) ||
      (write_cache && (((uintptr_t)q & 15) || (q_stride & 7) || (wq == nullptr) != (wk == nullptr))))
    return HB_BAD_ARGUMENT;
  AttnOptions opt = {};
  opt.sink = sink; opt.sink_values = sink_values;
  opt.gate = (const __nv_bfloat16*)gate; opt.gate_stride = gate_stride; opt.gate_wide = gate_wide;
  const QkPrepare prep = {wq, wk, eps, 0.f, 0};
  const PooledKeys pk = {(const __nv_bfloat16*)pooled_k, (const __nv_bfloat16*)pooled_v, pooled_table, pooled_stride,
                         pool, hd, vd, out_stride, factor};
  return pooled_dispatch(hd, vd, [&](auto H, auto V) {
    return launch_decode<decltype(H)::value, decltype(V)::value, POOLED_WARPS, true>(
        out, part_o, part_ml, q, q_stride, k_pages, v_pages, block_table, bt_stride, positions, S, nh, nkv, page_size,
        window, scale, n_splits, nullptr, nullptr, write_cache, opt, prep, pk, stream);
  });
}

HB_EXPORT int hb_attention_pooled_max_clusters(int hd, int vd, int cluster_size) {
  if (!pooled_sizes_ok(hd, vd) || cluster_size < 1 || cluster_size > 8) return -1;
  return pooled_dispatch(hd, vd, [&](auto H, auto V) {
    return decode_max_clusters<decltype(H)::value, decltype(V)::value, POOLED_WARPS, true>(cluster_size);
  });
}
