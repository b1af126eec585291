// bfloat16 attention over the paged cache on the tensor cores (mma.sync m16n8k16,
// float32 accumulate), for head sizes 32, 64, 96 and 128.
//
//   * decode: one query token per request.  A block takes one (request, KV head,
//     slice of the context); the query heads that share the KV head are the rows
//     of one MMA tile, so every key and value is read once for the whole group.
//     Up to 8 slices run as one thread-block cluster and are merged through distributed
//     shared memory; more are merged by a second kernel (flash-decoding).  A block has 4
//     or 8 warps, each with key tiles of its own.  The kernel can take the
//     step's rotary position encoding and cache write with it: every block rotates its
//     query heads in registers, and the one warp whose tile holds the request's new
//     token rotates that key and puts it and the value into the cache first
//     (python/helios/exec/model.py:148-153, paged_attn.py:74-85), which saves a launch.
//   * prefill / mixed: tiles of query tokens of one request against the keys the
//     cache holds for it, causal by position (and a window), whatever mix of
//     prompt portions and single tokens the batch is.
//
// Math follows python/helios/exec/paged_attn.py:264-408 (scores = q.k * scale, mask,
// softmax in float32, times V); pages are [page, kv head, slot, head_dim] as in
// paged_attn.py:49.  Scores, the running maximum, the sum and the output
// accumulators are float32; probabilities are rounded to bfloat16 for the PV
// product, as the reference casts them to the value dtype (paged_attn.py:293).
#include "common.cuh"
#include "attention_mma.cuh"
#include "attention_options.cuh"
#include "attention_decode.cuh"

namespace {

// ------------------------------------------------------------------------ prefill / mixed
constexpr int PRE_WARPS = 8;
constexpr int PRE_TILE = 64;   // keys per block tile

template <int HD>
__global__ void __launch_bounds__(PRE_WARPS * 32)
prefill_attention_kernel(__nv_bfloat16* __restrict__ out, const __nv_bfloat16* __restrict__ q,
                         int q_stride, const __nv_bfloat16* __restrict__ k_pages,
                         const __nv_bfloat16* __restrict__ v_pages,
                         const int* __restrict__ block_table, int bt_stride,
                         const int* __restrict__ q_tiles, const int* __restrict__ cu_tokens,
                         const int* __restrict__ start_pos, int nh, int nkv, int heads_per_block,
                         int token_subtiles, int page_size, int window, float scale_log2,
                         AttnOptions opt) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int RS = HD + 8;
  constexpr int TILE_ELEMS = PRE_TILE * RS;
  constexpr int CHUNKS = HD / 8;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __nv_bfloat16* smem = reinterpret_cast<__nv_bfloat16*>(smem_raw);   // [stage][k|v][tile]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int G = nh / nkv;
  const int head_blocks = (G + heads_per_block - 1) / heads_per_block;
  const int kvh = blockIdx.y / head_blocks, hb = blockIdx.y - kvh * head_blocks;
  const int seq = q_tiles[2 * blockIdx.x], t0 = q_tiles[2 * blockIdx.x + 1];
  const int tok0 = cu_tokens[seq], n_tok = cu_tokens[seq + 1] - tok0;
  if (t0 >= n_tok) return;      // padding of a captured step's tile list
  const int sp = start_pos[seq];
  const int BQ = 16 * token_subtiles;
  const int p_first = sp + t0;
  const int p_last = sp + min(n_tok, t0 + BQ) - 1;
  const int k_min = (window > 0 && p_first - window + 1 > 0) ? p_first - window + 1 : 0;
  // the first keys a window keeps: their tiles come before the window's
  const int keep = window > 0 ? opt.keep_first : 0;
  const int* table = block_table + (size_t)seq * bt_stride;

  const int head_local = warp % heads_per_block, sub = warp / heads_per_block;
  const int g_in_kv = hb * heads_per_block + head_local;
  const bool active = sub < token_subtiles && g_in_kv < G && (t0 + sub * 16) < n_tok;
  const int h = kvh * G + g_in_kv;
  const float head_slope_log2 = (opt.slopes != nullptr && g_in_kv < G) ? opt.slopes[h] * LOG2E : 0.f;
  const int g0 = lane >> 2, c0 = 2 * (lane & 3);
  // the two rows of this thread: local tokens and their positions
  const int tl0 = t0 + sub * 16 + g0, tl1 = tl0 + 8;
  const int pr0 = sp + tl0, pr1 = sp + tl1;

  uint32_t qa[HD / 16][4];
#pragma unroll
  for (int ks = 0; ks < HD / 16; ++ks) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int tl = (e & 1) ? tl1 : tl0;
      const int col = ks * 16 + c0 + (e >> 1) * 8;
      qa[ks][e] = (active && tl < n_tok)
          ? *reinterpret_cast<const uint32_t*>(q + (size_t)(tok0 + tl) * q_stride + (size_t)h * HD + col)
          : 0u;
    }
  }

  auto load_tile = [&](int kt, int stage) {
    __nv_bfloat16* kd = smem + (size_t)(stage * 2) * TILE_ELEMS;
    __nv_bfloat16* vd = kd + TILE_ELEMS;
    for (int idx = threadIdx.x; idx < PRE_TILE * CHUNKS; idx += PRE_WARPS * 32) {
      const int row = idx / CHUNKS, c = idx - row * CHUNKS;
      const int key = kt * PRE_TILE + row;
      const bool valid = (key >= k_min || key < keep) && key <= p_last;
      size_t base = 0;
      if (valid) {
        const int page = table[key / page_size];
        base = (((size_t)page * nkv + kvh) * page_size + key % page_size) * HD + c * 8;
      }
      const int bytes = valid ? 16 : 0;
      cp_async16(kd + row * RS + c * 8, k_pages + base, bytes);
      cp_async16(vd + row * RS + c * 8, v_pages + base, bytes);
    }
  };

  float o[HD / 8][4];
#pragma unroll
  for (int i = 0; i < HD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};

  const int kt_begin = k_min / PRE_TILE, kt_end = p_last / PRE_TILE + 1;
  // the key range this warp's 16 rows can see
  const int w_pmin = sp + t0 + sub * 16, w_pmax = min(w_pmin + 15, p_last);
  const int w_kmin = (window > 0 && w_pmin - window + 1 > 0) ? w_pmin - window + 1 : 0;

  // tiles 0 .. kept_tiles - 1 hold kept first keys; then the window's, from kt_begin on
  const int kept_tiles = min((min(keep, k_min) + PRE_TILE - 1) / PRE_TILE, kt_begin);
  auto next_tile = [&](int kt) { return (kt + 1 == kept_tiles) ? kt_begin : kt + 1; };
  const int kt_first = kept_tiles > 0 ? 0 : kt_begin;
  load_tile(kt_first, 0);
  cp_async_commit();
  int stage = 0;
  for (int kt = kt_first; kt < kt_end; kt = next_tile(kt), stage ^= 1) {
    if (next_tile(kt) < kt_end) load_tile(next_tile(kt), stage ^ 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const int key_base = kt * PRE_TILE;
    if (active && key_base <= w_pmax && (key_base + PRE_TILE - 1 >= w_kmin || key_base < keep)) {
      const __nv_bfloat16* ktile = smem + (size_t)(stage * 2) * TILE_ELEMS;
      const __nv_bfloat16* vtile = ktile + TILE_ELEMS;
      float s[PRE_TILE / 8][4];
#pragma unroll
      for (int i = 0; i < PRE_TILE / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
      qk_tile<HD, PRE_TILE / 8>(s, qa, ktile, lane);
#pragma unroll
      for (int nt = 0; nt < PRE_TILE / 8; ++nt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int key = key_base + nt * 8 + c0 + (e & 1);
          const int pr = (e >> 1) ? pr1 : pr0;
          const bool ok = key <= pr && (window <= 0 || key > pr - window || key < keep);
          if (opt.bias_table != nullptr)
            s[nt][e] = ok ? fmaf(s[nt][e], scale_log2, attn_table_bias_log2(opt, pr - key, h, nh)) : -INFINITY;
          else if (opt.slopes != nullptr)
            s[nt][e] = ok ? fmaf(s[nt][e], scale_log2, -head_slope_log2 * (float)(pr - key)) : -INFINITY;
          else
            s[nt][e] = ok ? s[nt][e] * scale_log2 : -INFINITY;
        }
      }
      softmax_step<HD, PRE_TILE / 8>(s, m, l, o);
      pv_tile<HD, PRE_TILE / 8>(o, s, vtile, lane);
    }
    __syncthreads();
  }
  cp_async_wait<0>();
  if (!active) return;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int tl = r ? tl1 : tl0;
    if (tl >= n_tok) continue;
    // attn_finish(1, m, l, ...) is the factor on every value of the row (1 / l without options)
    const float inv = attn_finish(1.f, m[r], l[r], opt.sink,
                                  opt.gate_wide ? 1.f : attn_gate_factor(opt, tok0 + tl, h), attn_sink_log2(opt, h));
    __nv_bfloat16* orow = out + ((size_t)(tok0 + tl) * nh + h) * HD;
#pragma unroll
    for (int nt = 0; nt < HD / 8; ++nt) {
      float g0v = 1.f, g1v = 1.f;
      if (opt.gate_wide) {
        g0v = attn_gate_factor(opt, tok0 + tl, h, nt * 8 + c0, HD);
        g1v = attn_gate_factor(opt, tok0 + tl, h, nt * 8 + c0 + 1, HD);
      }
      *reinterpret_cast<uint32_t*>(orow + nt * 8 + c0) =
          pack_bf16(o[nt][2 * r] * inv * g0v, o[nt][2 * r + 1] * inv * g1v);
    }
  }
}

template <int HD>
int launch_prefill(void* out, const void* q, int q_stride, const void* k_pages, const void* v_pages,
                   const int* block_table, int bt_stride, const int* q_tiles, int n_tiles,
                   const int* cu_tokens, const int* start_pos, int nh, int nkv, int heads_per_block,
                   int token_subtiles, int page_size, int window, float scale, AttnOptions opt,
                   cudaStream_t stream) {
  constexpr int RS = HD + 8;
  const size_t smem = (size_t)4 * PRE_TILE * RS * sizeof(__nv_bfloat16);
  auto kernel = prefill_attention_kernel<HD>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return HB_LAUNCH_FAILED;
    configured = true;
  }
  const int G = nh / nkv;
  const int head_blocks = (G + heads_per_block - 1) / heads_per_block;
  dim3 grid(n_tiles, nkv * head_blocks);
  hb_launch(kernel, dim3(grid), dim3(PRE_WARPS * 32), smem, stream, 
      (__nv_bfloat16*)out, (const __nv_bfloat16*)q, q_stride, (const __nv_bfloat16*)k_pages,
      (const __nv_bfloat16*)v_pages, block_table, bt_stride, q_tiles, cu_tokens, start_pos, nh, nkv,
      heads_per_block, token_subtiles, page_size, window, scale * LOG2E, opt);
  return hb_check_launch();
}

}  // namespace

#define HB_DISPATCH_HD(hd, ...)                         \
  switch (hd) {                                         \
    case 32: { constexpr int HD = 32; __VA_ARGS__; }    \
    case 64: { constexpr int HD = 64; __VA_ARGS__; }    \
    case 96: { constexpr int HD = 96; __VA_ARGS__; }    \
    case 128: { constexpr int HD = 128; __VA_ARGS__; }  \
    default: return HB_BAD_ARGUMENT;                    \
  }

// Decode: S requests, one token each (token i belongs to request i).  Needs the group
// size nh / nkv <= 16.  part_o: float [S, nh, n_splits, hd], part_ml: float
// [S, nh, n_splits, 2]; both unused when n_splits == 1.  With 2..8 slices and part_o null
// the slices run as one thread-block cluster and are merged through distributed shared
// memory instead of a second kernel.
//   q is a row of q|k|v per request ([nh + 2 nkv] heads, q_stride elements apart).  With
//   rot_cos / rot_sin (float [S, hd / 2]) the query heads are rotated on the way in (rotate-half
//   pairs (j, j + hd / 2)); with write_cache the request's key (rotated likewise) and value are
//   taken from that row and stored at its position in the pages before the kernel attends.
//   Without either, q must be rotated and the cache written already.
HB_EXPORT int hb_attention_decode_bf16(void* out, float* part_o, float* part_ml, const void* q,
                                       int q_stride, const void* k_pages, const void* v_pages,
                                       const int* block_table, int bt_stride, const int* positions,
                                       int S, int nh, int nkv, int hd, int page_size, int window,
                                       float scale, int n_splits, const float* rot_cos,
                                       const float* rot_sin, int write_cache, int warps,
                                       const float* slopes, int sink, const void* gate,
                                       int gate_stride, const float* bias_table, int bias_rows,
                                       const float* sink_values, int keep_first, int gate_wide,
                                       const float* norm_wq, const float* norm_wk,
                                       float norm_eps, float temp_coef, int temp_every,
                                       cudaStream_t stream) {
  if (S <= 0) return HB_OK;
  if (keep_first < 0 || (bias_table != nullptr && bias_rows <= 0)) return HB_BAD_ARGUMENT;
  const AttnOptions opt = {slopes, (const __nv_bfloat16*)gate, gate_stride, sink, bias_table, bias_rows,
                           sink_values, window > 0 ? keep_first : 0, gate_wide};
  const QkPrepare prep = {norm_wq, norm_wk, norm_eps, temp_coef, temp_every};
  if ((write_cache && (norm_wq == nullptr) != (norm_wk == nullptr)) || temp_every < 0) return HB_BAD_ARGUMENT;
  if (norm_wk != nullptr && !write_cache) return HB_BAD_ARGUMENT;     // a cached key is normed already
  if (nkv <= 0 || nh % nkv != 0 || nh / nkv > 16 || page_size <= 0 || n_splits < 1 ||
      (warps != 4 && warps != 8))
    return HB_BAD_ARGUMENT;
  if ((rot_cos == nullptr) != (rot_sin == nullptr)) return HB_BAD_ARGUMENT;
  if (write_cache && (q_stride < (nh + 2 * nkv) * hd || (q_stride & 7) || ((uintptr_t)q & 15)))
    return HB_BAD_ARGUMENT;
#define HB_DECODE(W)                                                                              \
  HB_DISPATCH_HD(hd, return (launch_decode<HD, HD, W, false>(out, part_o, part_ml, q, q_stride, k_pages, v_pages, \
                                                  block_table, bt_stride, positions, S, nh, nkv,      \
                                                  page_size, window, scale, n_splits, rot_cos,        \
                                                  rot_sin, write_cache, opt, prep, PooledKeys{}, stream)))
  if (warps == 8) HB_DECODE(8);
  HB_DECODE(4);
#undef HB_DECODE
}

HB_EXPORT int hb_attention_decode_max_clusters(int hd, int cluster_size, int warps) {
  if (cluster_size < 1 || cluster_size > 8 || (warps != 4 && warps != 8)) return -1;
  if (warps == 8) HB_DISPATCH_HD(hd, return (decode_max_clusters<HD, HD, 8, false>(cluster_size)));
  HB_DISPATCH_HD(hd, return (decode_max_clusters<HD, HD, 4, false>(cluster_size)));
}

// Prefill / mixed: q_tiles holds (request, first local token) for every tile of
// 16 * token_subtiles query tokens; heads_per_block * token_subtiles <= 8.
HB_EXPORT int hb_attention_prefill_bf16(void* out, const void* q, int q_stride, const void* k_pages,
                                        const void* v_pages, const int* block_table, int bt_stride,
                                        const int* q_tiles, int n_tiles, const int* cu_tokens,
                                        const int* start_pos, int nh, int nkv, int hd,
                                        int heads_per_block, int token_subtiles, int page_size,
                                        int window, float scale, const float* slopes, int sink,
                                        const void* gate, int gate_stride, const float* bias_table,
                                        int bias_rows, const float* sink_values, int keep_first,
                                        int gate_wide, cudaStream_t stream) {
  if (n_tiles <= 0) return HB_OK;
  if (keep_first < 0 || (bias_table != nullptr && bias_rows <= 0)) return HB_BAD_ARGUMENT;
  const AttnOptions opt = {slopes, (const __nv_bfloat16*)gate, gate_stride, sink, bias_table, bias_rows,
                           sink_values, window > 0 ? keep_first : 0, gate_wide};
  if (nkv <= 0 || nh % nkv != 0 || page_size <= 0 || heads_per_block < 1 || token_subtiles < 1 ||
      heads_per_block * token_subtiles > PRE_WARPS)
    return HB_BAD_ARGUMENT;
  HB_DISPATCH_HD(hd, return launch_prefill<HD>(out, q, q_stride, k_pages, v_pages, block_table,
                                               bt_stride, q_tiles, n_tiles, cu_tokens, start_pos,
                                               nh, nkv, heads_per_block, token_subtiles, page_size,
                                               window, scale, opt, stream));
}
