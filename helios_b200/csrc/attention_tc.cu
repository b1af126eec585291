// Prefill attention on the 5th-generation tensor cores (attention_prefill_tc.cuh) for values of
// the keys' size, 64 or 128.
#include "attention_prefill_tc.cuh"

namespace {

template <int HD>
int launch_tc(const AttnArgs& a, const void* k_pages, const void* v_pages, long long page_rows, int n_tiles,
              cudaStream_t stream) {
  constexpr size_t SMEM = TcStages<HD, HD>::BYTES;
  CUtensorMap map_k, map_v;
  if (!make_map(&map_k, k_pages, (uint64_t)page_rows, HD, HD, a.page_size)) return HB_LAUNCH_FAILED;
  if (!make_map(&map_v, v_pages, (uint64_t)page_rows, HD, HD, a.page_size)) return HB_LAUNCH_FAILED;
  auto kernel = attention_prefill_tc_kernel<HD, HD, false>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM) != cudaSuccess)
      return HB_LAUNCH_FAILED;
    configured = true;
  }
  hb_launch(kernel, dim3(n_tiles * a.nkv), dim3(TC_THREADS), SMEM, stream, map_k, map_v, map_k, map_v, a, PooledTiles{});
  return hb_check_launch();
}

}  // namespace

// q_tiles: (request, first local token) for tiles of 128 / (nh / nkv) tokens.  Needs hd in
// {64, 128}, a group size that divides 128, and a page size that is a multiple of 8 and
// divides 128.  num_pages: pages in k_pages / v_pages ([pages, nkv, page_size, hd]).
// bias_table_t: the bias by distance as float [nh, bias_rows] (the transpose of what the
// other attention kernels take).
HB_EXPORT int hb_attention_prefill_tc(void* out, const void* q, int q_stride, const void* k_pages,
                                      const void* v_pages, long long num_pages, const int* block_table,
                                      int bt_stride, const int* q_tiles, int n_tiles, const int* cu_tokens,
                                      const int* start_pos, int nh, int nkv, int hd, int page_size, int window,
                                      float scale, int* error, const float* slopes, int sink,
                                      const void* gate, int gate_stride, const float* bias_table_t,
                                      int bias_rows, const float* sink_values, int keep_first, int gate_wide,
                                      cudaStream_t stream) {
  if (n_tiles <= 0) return HB_OK;
  if (nkv <= 0 || nh % nkv != 0 || error == nullptr) return HB_BAD_ARGUMENT;
  if (keep_first < 0 || (bias_table_t != nullptr && bias_rows <= 0)) return HB_BAD_ARGUMENT;
  const int G = nh / nkv;
  if (G > TILE) return HB_BAD_ARGUMENT;
  if (page_size < 8 || page_size % 8 != 0 || TILE % page_size != 0) return HB_BAD_ARGUMENT;
  if (((uintptr_t)q & 15) || ((uintptr_t)k_pages & 15) || ((uintptr_t)v_pages & 15) || (q_stride & 7))
    return HB_BAD_ARGUMENT;
  AttnArgs a;
  a.out = (__nv_bfloat16*)out; a.q = (const __nv_bfloat16*)q; a.q_stride = q_stride;
  a.block_table = block_table; a.bt_stride = bt_stride; a.q_tiles = q_tiles; a.cu_tokens = cu_tokens;
  a.start_pos = start_pos; a.nh = nh; a.nkv = nkv; a.page_size = page_size; a.window = window;
  a.scale_log2 = scale * LOG2E; a.error = error;
  a.opt = AttnOptions{slopes, (const __nv_bfloat16*)gate, gate_stride, sink, nullptr, bias_rows, sink_values,
                      window > 0 ? keep_first : 0, gate_wide};
  a.bias_t = bias_table_t;
  const long long rows = num_pages * nkv * page_size;
  if (hd == 128) return launch_tc<128>(a, k_pages, v_pages, rows, n_tiles, stream);
  if (hd == 64) return launch_tc<64>(a, k_pages, v_pages, rows, n_tiles, stream);
  return HB_BAD_ARGUMENT;
}
