// Prefill attention on the 5th-generation tensor cores (attention_prefill_tc.cuh) with keys and values
// of sizes of their own up to 256 (not both above 128), compiled for 64, 128 and 256 each: over a
// window's tokens and the means of whole blocks behind it, under one softmax, or over all tokens or a
// window's without such blocks; with a sink and a gate.  The keys and values of a step may also lie in
// rows of their own instead of pages a head (hb_attention_rows_prefill_tc).
#include <type_traits>
#include "attention_prefill_tc.cuh"

namespace {

// k_pages / v_pages: page_rows rows, k_ld / v_ld elements apart, of k_cols / v_cols columns.
template <int HD, int VD>
int launch_maps(const AttnArgs& a, const PooledTiles& pl, const void* k_pages, const void* v_pages,
                long long page_rows, int k_cols, int k_ld, int v_cols, int v_ld, const void* pooled_k, const void* pooled_v, long long pooled_rows, int n_tiles,
                  cudaStream_t stream) {
  constexpr size_t SMEM = TcStages<HD, VD>::BYTES;
  CUtensorMap map_k, map_v, map_pk, map_pv;
  if (!make_map(&map_k, k_pages, (uint64_t)page_rows, k_cols, k_ld, a.page_size) ||
      !make_map(&map_v, v_pages, (uint64_t)page_rows, v_cols, v_ld, a.page_size))
    return HB_LAUNCH_FAILED;
  map_pk = map_k;
  map_pv = map_v;
  if (pl.pool > 0 && (!make_map(&map_pk, pooled_k, (uint64_t)pooled_rows, pl.hd, pl.hd, a.page_size) ||
                      !make_map(&map_pv, pooled_v, (uint64_t)pooled_rows, pl.vd, pl.vd, a.page_size)))
    return HB_LAUNCH_FAILED;
  auto kernel = attention_prefill_tc_kernel<HD, VD, true>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM) != cudaSuccess)
      return HB_LAUNCH_FAILED;
    configured = true;
  }
  hb_launch(kernel, dim3(n_tiles * a.nkv), dim3(TC_THREADS), SMEM, stream, map_k, map_v, map_pk, map_pv, a, pl);
  return hb_check_launch();
}

template <typename F>
int dispatch_sizes(int hd, int vd, F f) {
  auto values = [&](auto H) {
    if (vd <= 64) return f(H, std::integral_constant<int, 64>());
    if (vd <= 128) return f(H, std::integral_constant<int, 128>());
    if constexpr (decltype(H)::value <= 128) return f(H, std::integral_constant<int, 256>());
    else return (int)HB_BAD_ARGUMENT;
  };
  if (hd <= 64) return values(std::integral_constant<int, 64>());
  if (hd <= 128) return values(std::integral_constant<int, 128>());
  if (hd <= 192) return values(std::integral_constant<int, 192>());
  return values(std::integral_constant<int, 256>());
}

}  // namespace

// q [T, nh * hd]; q_tiles: (request, first local token) for tiles of 128 / (nh / nkv) tokens.  Page
// sizes that are multiples of 8 and divide 128.  num_pages / pooled_num_pages: pages of the tokens'
// and the blocks' keys and values.
HB_EXPORT int hb_attention_pooled_prefill_tc(void* out, int out_stride, float factor, const void* q, int q_stride,
                                             const void* k_pages, const void* v_pages, long long num_pages,
                                             const int* block_table, int bt_stride, const void* pooled_k,
                                             const void* pooled_v, long long pooled_num_pages,
                                             const int* pooled_table, int pooled_stride, int pool, const int* q_tiles,
                                             int n_tiles, const int* cu_tokens, const int* start_pos, int nh, int nkv,
                                             int hd, int vd, int page_size, int window, float scale, int* error,
                                             int sink, const float* sink_values, const void* gate, int gate_stride,
                                             int gate_wide, cudaStream_t stream) {
  if (n_tiles <= 0) return HB_OK;
  if (nkv <= 0 || nh % nkv != 0 || nh / nkv > TILE || error == nullptr || hd <= 0 || hd > 256 || hd % 8 || vd <= 0 ||
      vd > 256 || vd % 8 || (hd > 128 && vd > 128) || window < 0 || pool < 0 || (pool > 0 && window <= 0) || page_size < 8 || page_size % 8 != 0 ||
      TILE % page_size != 0 || (q_stride & 7) || (out_stride & 7) || out_stride < nh * vd ||
      (pool > 0 && (!pooled_k || !pooled_v || !pooled_table)) ||
      (((uintptr_t)q | (uintptr_t)out | (uintptr_t)k_pages | (uintptr_t)v_pages | (uintptr_t)pooled_k |
        (uintptr_t)pooled_v) & 15))
    return HB_BAD_ARGUMENT;
  AttnArgs a = {};
  a.out = (__nv_bfloat16*)out; a.q = (const __nv_bfloat16*)q; a.q_stride = q_stride;
  a.block_table = block_table; a.bt_stride = bt_stride; a.q_tiles = q_tiles; a.cu_tokens = cu_tokens;
  a.start_pos = start_pos; a.nh = nh; a.nkv = nkv; a.page_size = page_size; a.window = window;
  a.scale_log2 = scale * LOG2E; a.error = error;
  a.opt.sink = sink; a.opt.sink_values = sink_values;
  a.opt.gate = (const __nv_bfloat16*)gate; a.opt.gate_stride = gate_stride; a.opt.gate_wide = gate_wide;
  const PooledTiles pl = {pooled_table, pooled_stride, pool, hd, vd, out_stride, factor, 0};
  const long long rows = num_pages * nkv * page_size, prows = pooled_num_pages * nkv * page_size;
  return dispatch_sizes(hd, vd, [&](auto H, auto V) {
    return launch_maps<decltype(H)::value, decltype(V)::value>(a, pl, k_pages, v_pages, rows, hd, hd, vd, vd, pooled_k,
                                                               pooled_v, prows, n_tiles, stream);
  });
}

// The same attention with keys and values in rows: kv [rows, ld] holds a token's keys [heads * hd] and
// behind them its values [heads * vd]; `table` counts pages of page_size such rows.  Every head has keys
// and values of its own.
HB_EXPORT int hb_attention_rows_prefill_tc(void* out, int out_stride, const void* q, int q_stride, const void* kv,
                                           int ld, long long rows, const int* table, int table_stride,
                                           const int* q_tiles, int n_tiles, const int* cu_tokens, const int* start_pos,
                                           int heads, int hd, int vd, int page_size, int window, float scale,
                                           int* error, int sink, const float* sink_values, const void* gate,
                                           int gate_stride, int gate_wide, cudaStream_t stream) {
  if (n_tiles <= 0) return HB_OK;
  if (heads <= 0 || error == nullptr || hd <= 0 || hd > 256 || hd % 8 || vd <= 0 || vd > 256 || vd % 8 ||
      (hd > 128 && vd > 128) || window < 0 || page_size < 8 || page_size % 8 != 0 || TILE % page_size != 0 ||
      (q_stride & 7) || (out_stride & 7) || out_stride < heads * vd || (ld & 7) || ld < heads * (hd + vd) ||
      (((uintptr_t)q | (uintptr_t)out | (uintptr_t)kv) & 15))
    return HB_BAD_ARGUMENT;
  AttnArgs a = {};
  a.out = (__nv_bfloat16*)out; a.q = (const __nv_bfloat16*)q; a.q_stride = q_stride;
  a.block_table = table; a.bt_stride = table_stride; a.q_tiles = q_tiles; a.cu_tokens = cu_tokens;
  a.start_pos = start_pos; a.nh = heads; a.nkv = heads; a.page_size = page_size; a.window = window;
  a.scale_log2 = scale * LOG2E; a.error = error;
  a.opt.sink = sink; a.opt.sink_values = sink_values;
  a.opt.gate = (const __nv_bfloat16*)gate; a.opt.gate_stride = gate_stride; a.opt.gate_wide = gate_wide;
  const PooledTiles pl = {nullptr, 0, 0, hd, vd, out_stride, 1.f, 1};
  const __nv_bfloat16* k = (const __nv_bfloat16*)kv;
  return dispatch_sizes(hd, vd, [&](auto H, auto V) {
    return launch_maps<decltype(H)::value, decltype(V)::value>(a, pl, k, k + (size_t)heads * hd, rows, heads * hd, ld,
                                                               heads * vd, ld, nullptr, nullptr, 0, n_tiles, stream);
  });
}
