// Decode attention over the paged cache on the tensor cores (mma.sync m16n8k16, bfloat16
// operands, float32 accumulators): one query token per request.  A block takes one (request, KV
// head, slice of the context); the query heads that share the KV head are the rows of one MMA
// tile, so every key and value is read once for the whole group.  Up to 8 slices run as one
// thread-block cluster and are merged through distributed shared memory; more are merged by a
// second kernel.  Compiled by attention_bf16.cu (values of the keys' size) and attention_pooled.cu
// (values of a size of their own, means of whole blocks behind the window).
#pragma once
#include <type_traits>
#include "common.cuh"
#include "attention_mma.cuh"
#include "attention_options.cuh"

namespace {

// ------------------------------------------------------------------------ decode
// (warps per decode block, a template parameter: 4, two blocks an SM, or 8, one block an SM,
// where so few blocks run that each warp's chain of key tiles, not the memory, bounds the kernel)
constexpr int DEC_TILE = 16;      // keys per warp tile
constexpr int DEC_STAGES = 3;     // tiles a warp keeps in shared memory (all but one in flight)

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// The online-softmax step of the decode kernel over a tile's scaled, masked scores (log2
// domain).  Without WIDE only the first eight rows of the MMA tile are query heads: the
// second row group (rows 8-15, zero queries) is left out and its probabilities are zero.
// The output and the sum are rescaled only in tiles where some row's maximum grew (a
// warp-wide vote; otherwise every factor would be exactly 1).
template <int HD, int NT, bool WIDE>
__device__ __forceinline__ void decode_softmax_step(float (&s)[NT][4], float (&m)[2], float (&l)[2],
                                                    float (&o)[HD / 8][4]) {
  constexpr int R = WIDE ? 2 : 1;
  float m_new[2] = {m[0], m[1]};
  bool grew = false;
#pragma unroll
  for (int r = 0; r < R; ++r) {
    float mx = -INFINITY;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) mx = fmaxf(mx, fmaxf(s[nt][2 * r], s[nt][2 * r + 1]));
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
    m_new[r] = fmaxf(m[r], mx);
    grew = grew || m_new[r] > m[r];
  }
  if (__any_sync(0xffffffffu, grew)) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const float corr = fast_exp2(m[r] - ((m_new[r] == -INFINITY) ? 0.f : m_new[r]));
      l[r] *= corr;
#pragma unroll
      for (int nt = 0; nt < HD / 8; ++nt) {
        o[nt][2 * r] *= corr;
        o[nt][2 * r + 1] *= corr;
      }
    }
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    m[r] = m_new[r];
    const float m_use = (m_new[r] == -INFINITY) ? 0.f : m_new[r];
    float sum = 0.f;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      s[nt][2 * r] = fast_exp2(s[nt][2 * r] - m_use);
      s[nt][2 * r + 1] = fast_exp2(s[nt][2 * r + 1] - m_use);
      sum += s[nt][2 * r] + s[nt][2 * r + 1];
    }
    l[r] += sum;
  }
  if (!WIDE) {
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) s[nt][2] = s[nt][3] = 0.f;
  }
}

// Means of whole blocks of `pool` tokens behind the window, a key and a value each in pages of
// their own ([page, kv head, slot, size]), for a kernel compiled with POOLED; block b is seen at
// position p if (b + 1) * pool <= p - window + 1.  Such a kernel also takes key and value sizes
// (multiples of 8) below the ones it is compiled for, rows of the output that are out_stride
// apart, and a constant factor on the output.
struct PooledKeys {
  const __nv_bfloat16* k;
  const __nv_bfloat16* v;
  const int* table;
  int table_stride;
  int pool;                 // 0: no blocks
  int hd, vd;
  int out_stride;
  float factor;
};

template <int HD, int VD, int WARPS, bool POOLED>
__global__ void __launch_bounds__(WARPS * 32)
decode_attention_kernel(__nv_bfloat16* __restrict__ out, float* __restrict__ part_o,
                        float* __restrict__ part_ml, const __nv_bfloat16* __restrict__ q,
                        int q_stride, const __nv_bfloat16* __restrict__ k_pages,
                        const __nv_bfloat16* __restrict__ v_pages,
                        const int* __restrict__ block_table, int bt_stride,
                        const int* __restrict__ positions, int nh, int nkv, int page_size,
                        int window, float scale_log2, int n_splits, int cluster_merge,
                        const float* __restrict__ rot_cos, const float* __restrict__ rot_sin,
                        __nv_bfloat16* k_write, __nv_bfloat16* v_write, AttnOptions opt,
                        QkPrepare prep, PooledKeys pk) {
  // rot_cos / rot_sin [requests, HD / 2]: q (and the new key) still lack their rotation.
  // k_write / v_write (the cache again, writable): the new token's key and value are still
  // in the q|k|v row and go into the cache here.
  pdl_launch_dependents();
  static_assert(POOLED || HD == VD, "values of another size come with the pooled kernels");
  constexpr int RS = HD + 8, RSV = VD + 8;
  constexpr int TILE_ELEMS = DEC_TILE * RS, STAGE_ELEMS = TILE_ELEMS + DEC_TILE * RSV;
  const int hd = POOLED ? pk.hd : HD, vd = POOLED ? pk.vd : VD;
  const int out_stride = POOLED ? pk.out_stride : nh * HD;
  const float out_factor = POOLED ? pk.factor : 1.f;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __nv_bfloat16* smem = reinterpret_cast<__nv_bfloat16*>(smem_raw);

  const int split = blockIdx.x, kvh = blockIdx.y, seq = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int G = nh / nkv;
  const int pos = positions[seq];
  const int lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
  // Tiles start at a multiple of the tile size where pages hold whole tiles: then every tile's
  // keys are consecutive slots of ONE page.  Keys of the first tile from before the window
  // are zero-filled and masked.
  const bool whole_pages = page_size % DEC_TILE == 0;
  const int first = whole_pages ? lo - lo % DEC_TILE : lo;
  const int n_keys = pos - first + 1;
  // The first keys a window keeps (those it has passed) come as tiles of their own BEFORE the
  // window's: tile t < kept_tiles holds the keys from t * DEC_TILE on, valid below kept_end.
  // With POOLED the blocks behind the window take that place, from pages of their own.
  const int kept_end = POOLED ? (pk.pool > 0 ? lo / pk.pool : 0)
                              : (window > 0 && opt.keep_first > 0) ? min(opt.keep_first, lo) : 0;
  const int kept_tiles = (kept_end + DEC_TILE - 1) / DEC_TILE;
  // slices of whole tiles
  const int tiles_total = kept_tiles + (n_keys + DEC_TILE - 1) / DEC_TILE;
  const int tiles_per_split = (tiles_total + n_splits - 1) / n_splits;
  const int tile_begin = split * tiles_per_split;
  const int tile_end = min(tiles_total, tile_begin + tiles_per_split);
  const int k_end = pos + 1;
  // slopes of the distance bias for this thread's two rows of the tile (heads g0 and g0 + 8)
  float slope_log2[2] = {0.f, 0.f};
  if (opt.slopes != nullptr) {
    const int g0 = lane >> 2;
    if (g0 < G) slope_log2[0] = opt.slopes[kvh * G + g0] * LOG2E;
    if (g0 + 8 < G) slope_log2[1] = opt.slopes[kvh * G + g0 + 8] * LOG2E;
  }
  const int* table = block_table + (size_t)seq * bt_stride;

  __nv_bfloat16* my = smem + (size_t)warp * DEC_STAGES * STAGE_ELEMS;   // [stage][k|v][tile]
  // A tile is DEC_TILE rows of HD/8 16-byte chunks; consecutive lanes copy consecutive
  // chunks, so a warp instruction reads 512 contiguous bytes.  Where the tile's keys are
  // consecutive slots of ONE page (page_size a multiple of the tile) the whole tile is one
  // contiguous stretch of the cache: one look-up in the block table and one address per
  // warp.  Otherwise lane r first finds the cache row of key r.
  auto load_tile = [&](int tile, int stage) {
    constexpr int CH = HD / 8, CHV = VD / 8;
    __nv_bfloat16* k_dst = my + (size_t)stage * STAGE_ELEMS;
    __nv_bfloat16* v_dst = k_dst + TILE_ELEMS;
    const bool kept = tile < kept_tiles;
    const int t_first = kept ? tile * DEC_TILE : first + (tile - kept_tiles) * DEC_TILE;
    const int t_end = kept ? kept_end : k_end, t_lo = kept ? 0 : lo;
    const bool blocks = POOLED && kept;
    const int* tab = blocks ? pk.table + (size_t)seq * pk.table_stride : table;
    const __nv_bfloat16* k_src = blocks ? pk.k : k_pages;
    const __nv_bfloat16* v_src = blocks ? pk.v : v_pages;
    if (whole_pages) {
      const int key_first = t_first;
      const int page = tab[key_first / page_size];
      const size_t row0 = (size_t)(page * nkv + kvh) * page_size + key_first % page_size;
      const int rows_valid = t_end - key_first;            // >= 1; rows from there on are zero-filled,
      const int rows_skipped = t_lo - key_first;           // and so are rows before the window
#pragma unroll
      for (int it = 0; it < DEC_TILE * CH / 32; ++it) {
        const int idx = it * 32 + lane;
        const int row = idx / CH, c = idx - row * CH;
        if constexpr (!POOLED) {         // the tile is one contiguous stretch of the cache
          const int bytes = (row < rows_valid && row >= rows_skipped) ? 16 : 0;
          const size_t base = row0 * HD + lane * 8;
          cp_async16(k_dst + row * RS + c * 8, k_pages + base + it * 256, bytes);
          cp_async16(v_dst + row * RS + c * 8, v_pages + base + it * 256, bytes);
        } else {
          const int bytes = (row < rows_valid && row >= rows_skipped && c * 8 < hd) ? 16 : 0;
          cp_async16(k_dst + row * RS + c * 8, k_src + (bytes ? (row0 + row) * hd + c * 8 : 0), bytes);
        }
      }
      if constexpr (POOLED) {
#pragma unroll
        for (int it = 0; it < DEC_TILE * CHV / 32; ++it) {
          const int idx = it * 32 + lane;
          const int row = idx / CHV, c = idx - row * CHV;
          const int bytes = (row < rows_valid && row >= rows_skipped && c * 8 < vd) ? 16 : 0;
          cp_async16(v_dst + row * RSV + c * 8, v_src + (bytes ? (row0 + row) * vd + c * 8 : 0), bytes);
        }
      }
      return;
    }
    int row_id = -1;
    if (lane < DEC_TILE) {
      const int key = t_first + lane;
      if (key < t_end) {
        const int page = tab[key / page_size];
        row_id = (page * nkv + kvh) * page_size + key % page_size;
      }
    }
#pragma unroll
    for (int it = 0; it < DEC_TILE * CH / 32; ++it) {
      const int idx = it * 32 + lane;
      const int row = idx / CH, c = idx - row * CH;
      const int rid = __shfl_sync(0xffffffffu, row_id, row);
      if constexpr (!POOLED) {
        const size_t base = (size_t)(rid < 0 ? 0 : rid) * HD + c * 8;
        const int bytes = rid < 0 ? 0 : 16;
        cp_async16(k_dst + row * RS + c * 8, k_pages + base, bytes);
        cp_async16(v_dst + row * RS + c * 8, v_pages + base, bytes);
      } else {
        const int bytes = (rid < 0 || c * 8 >= hd) ? 0 : 16;
        cp_async16(k_dst + row * RS + c * 8, k_src + (bytes ? (size_t)rid * hd + c * 8 : 0), bytes);
      }
    }
    if constexpr (POOLED) {
#pragma unroll
      for (int it = 0; it < DEC_TILE * CHV / 32; ++it) {
        const int idx = it * 32 + lane;
        const int row = idx / CHV, c = idx - row * CHV;
        const int rid = __shfl_sync(0xffffffffu, row_id, row);
        const int bytes = (rid < 0 || c * 8 >= vd) ? 0 : 16;
        cp_async16(v_dst + row * RSV + c * 8, v_src + (bytes ? (size_t)rid * vd + c * 8 : 0), bytes);
      }
    }
  };

  float o[VD / 8][4];
#pragma unroll
  for (int i = 0; i < VD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};

  // prologue: DEC_STAGES - 1 tiles in flight.  Keys of earlier steps do not depend on the
  // kernel before this one (the block tables and positions were copied before the step's
  // first kernel): their tiles are fetched while that kernel still runs.  The tile with
  // the token's own key, which that kernel writes, and the query follow after the wait.
  int tile = tile_begin + warp;
  bool early[DEC_STAGES - 1];
#pragma unroll
  for (int p = 0; p < DEC_STAGES - 1; ++p) {
    const int tp = tile + p * WARPS;
    early[p] = tp < tile_end && tp < tiles_total - 1;
    if (early[p]) load_tile(tp, p);
  }
  pdl_wait();
  {
    // the warp whose tile holds the request's own token (the last tile) writes its key and
    // value before it fetches that tile
    const int last_tile = tiles_total - 1;
    if (k_write != nullptr && last_tile >= tile_begin && last_tile < tile_end &&
        (last_tile - tile_begin) % WARPS == warp) {
      const int page = table[pos / page_size];
      const size_t row0 = (size_t)(page * nkv + kvh) * page_size + pos % page_size;
      const __nv_bfloat16* k_new = q + (size_t)seq * q_stride + (size_t)nh * hd + (size_t)kvh * hd;
      const __nv_bfloat16* v_new = q + (size_t)seq * q_stride + (size_t)(nh + nkv) * hd + (size_t)kvh * vd;
      if constexpr (POOLED) {
        // sizes of their own, no rotation: a lane holds every 32nd pair of the key
        __nv_bfloat16* kd = k_write + row0 * hd;
        float2 x[HD / 64];
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < HD / 64; ++i) {
          const int j = 2 * lane + 64 * i;
          x[i] = j < hd ? __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(k_new + j)) : make_float2(0.f, 0.f);
          ss += x[i].x * x[i].x + x[i].y * x[i].y;
        }
        const float f = prep.wk != nullptr ? rsqrtf(warp_sum(ss) / (float)hd + prep.eps) : 1.f;
#pragma unroll
        for (int i = 0; i < HD / 64; ++i) {
          const int j = 2 * lane + 64 * i;
          if (j >= hd) continue;
          const float2 w = prep.wk != nullptr ? *reinterpret_cast<const float2*>(prep.wk + j) : make_float2(1.f, 1.f);
          *reinterpret_cast<__nv_bfloat162*>(kd + j) = __floats2bfloat162_rn(x[i].x * f * w.x, x[i].y * f * w.y);
        }
        for (int j = 8 * lane; j < vd; j += 256)
          *reinterpret_cast<uint4*>(v_write + row0 * vd + j) = *reinterpret_cast<const uint4*>(v_new + j);
      } else {
        const size_t dst = row0 * HD;
        // a lane holds the pairs (j, j + 1) of both halves of the key: HD / 2 <= 64, one trip
        float k_factor = 1.f;
        if (prep.wk != nullptr) {
          float ss = 0.f;
          const int j = 2 * lane;
          if (j < HD / 2) {
            const float2 x1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(k_new + j));
            const float2 x2 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(k_new + j + HD / 2));
            ss = x1.x * x1.x + x1.y * x1.y + x2.x * x2.x + x2.y * x2.y;
          }
          k_factor = rsqrtf(warp_sum(ss) / (float)HD + prep.eps);
        }
        for (int j = 2 * lane; j < HD / 2; j += 64) {
          float2 x1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(k_new + j));
          float2 x2 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(k_new + j + HD / 2));
          if (prep.wk != nullptr) {
            const float2 w1 = *reinterpret_cast<const float2*>(prep.wk + j);
            const float2 w2 = *reinterpret_cast<const float2*>(prep.wk + j + HD / 2);
            x1 = make_float2(x1.x * k_factor * w1.x, x1.y * k_factor * w1.y);
            x2 = make_float2(x2.x * k_factor * w2.x, x2.y * k_factor * w2.y);
          }
          float2 r1 = x1, r2 = x2;
          if (rot_cos != nullptr) {
            const float2 c = *reinterpret_cast<const float2*>(rot_cos + (size_t)seq * (HD / 2) + j);
            const float2 sn = *reinterpret_cast<const float2*>(rot_sin + (size_t)seq * (HD / 2) + j);
            r1 = make_float2(x1.x * c.x - x2.x * sn.x, x1.y * c.y - x2.y * sn.y);
            r2 = make_float2(x2.x * c.x + x1.x * sn.x, x2.y * c.y + x1.y * sn.y);
          }
          *reinterpret_cast<__nv_bfloat162*>(k_write + dst + j) = __floats2bfloat162_rn(r1.x, r1.y);
          *reinterpret_cast<__nv_bfloat162*>(k_write + dst + j + HD / 2) = __floats2bfloat162_rn(r2.x, r2.y);
        }
        for (int j = 8 * lane; j < HD; j += 256)
          *reinterpret_cast<uint4*>(v_write + dst + j) = *reinterpret_cast<const uint4*>(v_new + j);
      }
      __syncwarp();           // the copies below, by other lanes, read these rows
    }
  }
#pragma unroll
  for (int p = 0; p < DEC_STAGES - 1; ++p) {
    const int tp = tile + p * WARPS;
    if (tp < tile_end && !early[p]) load_tile(tp, p);
    cp_async_commit();
  }

  // query fragments: rows = the group's heads (zero beyond G)
  uint32_t qa[HD / 16][4];
  {
    const int g0 = lane >> 2, c0 = 2 * (lane & 3);
    const __nv_bfloat16* qrow = q + (size_t)seq * q_stride + (size_t)kvh * G * hd;
#pragma unroll
    for (int ks = 0; ks < HD / 16; ++ks) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int row = g0 + (e & 1) * 8;
        const int col = ks * 16 + c0 + (e >> 1) * 8;
        qa[ks][e] = (row < G && col < hd) ? *reinterpret_cast<const uint32_t*>(qrow + (size_t)row * hd + col) : 0u;
      }
    }
    if (prep.wq != nullptr || prep.every > 0) {
      // a head's values are spread over the four lanes of a quad: rows g0 (e even) and g0 + 8
      float ss[2] = {0.f, 0.f};
#pragma unroll
      for (int ks = 0; ks < HD / 16; ++ks) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 x = __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&qa[ks][e]));
          ss[e & 1] += x.x * x.x + x.y * x.y;
        }
      }
      float inv_rms[2];
      const float temp = prep.every > 0 ? 1.f + prep.coef * logf((float)((pos + 1) / prep.every) + 1.f) : 1.f;
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 1);
        ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 2);
        inv_rms[r] = prep.wq != nullptr ? rsqrtf(ss[r] / (float)hd + prep.eps) : 1.f;
      }
#pragma unroll
      for (int ks = 0; ks < HD / 16; ++ks) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int col = ks * 16 + c0 + (e >> 1) * 8;
          const float2 w = prep.wq != nullptr && col < hd ? *reinterpret_cast<const float2*>(prep.wq + col)
                                                          : make_float2(1.f, 1.f);
          const float2 x = __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&qa[ks][e]));
          // the norm, the weight, then the temperature: the order of the kernel that does this alone
          const float f = inv_rms[e & 1];
          __nv_bfloat162 y = __floats2bfloat162_rn(x.x * f * w.x * temp, x.y * f * w.y * temp);
          qa[ks][e] = *reinterpret_cast<uint32_t*>(&y);
        }
      }
    }
    if (rot_cos != nullptr) {
      // rotate-half pairs (j, j + HD / 2): both values of a pair are in this thread's fragments
      const float* cs = rot_cos + (size_t)seq * (HD / 2);
      const float* sn = rot_sin + (size_t)seq * (HD / 2);
#pragma unroll
      for (int ks = 0; ks < HD / 32; ++ks) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int col = ks * 16 + c0 + (e >> 1) * 8;
          const float2 c = *reinterpret_cast<const float2*>(cs + col);
          const float2 sv = *reinterpret_cast<const float2*>(sn + col);
          const float2 x1 = __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&qa[ks][e]));
          const float2 x2 = __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&qa[ks + HD / 32][e]));
          __nv_bfloat162 r1 = __floats2bfloat162_rn(x1.x * c.x - x2.x * sv.x, x1.y * c.y - x2.y * sv.y);
          __nv_bfloat162 r2 = __floats2bfloat162_rn(x2.x * c.x + x1.x * sv.x, x2.y * c.y + x1.y * sv.y);
          qa[ks][e] = *reinterpret_cast<uint32_t*>(&r1);
          qa[ks + HD / 32][e] = *reinterpret_cast<uint32_t*>(&r2);
        }
      }
    }
  }

  // the key tiles of this warp; `wide` (a compile-time tag): more than eight query heads
  // share the KV head, so both row groups of the MMA tile are live
  auto run = [&](auto wide) {
    constexpr bool WIDE = decltype(wide)::value;
    int stage = 0;
    for (; tile < tile_end; tile += WARPS) {
      const int ahead = tile + (DEC_STAGES - 1) * WARPS;
      int put = stage + DEC_STAGES - 1;
      if (put >= DEC_STAGES) put -= DEC_STAGES;
      if (ahead < tile_end) load_tile(ahead, put);
      cp_async_commit();
      cp_async_wait<DEC_STAGES - 1>();
      __syncwarp();
      const __nv_bfloat16* kt = my + (size_t)stage * STAGE_ELEMS;
      const __nv_bfloat16* vt = kt + TILE_ELEMS;
      float s[DEC_TILE / 8][4];
#pragma unroll
      for (int i = 0; i < DEC_TILE / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
      qk_tile<HD, DEC_TILE / 8>(s, qa, kt, lane);
      const bool kept = tile < kept_tiles;
      const int tile_key0 = kept ? tile * DEC_TILE : first + (tile - kept_tiles) * DEC_TILE;
      const int t_end = kept ? kept_end : k_end, t_lo = kept ? 0 : lo;
      if (opt.bias_table != nullptr) {
        // a bias looked up by the distance, for every row (head) of the tile
        const int key0 = tile_key0 + 2 * (lane & 3);
        const int g0 = lane >> 2;
#pragma unroll
        for (int nt = 0; nt < DEC_TILE / 8; ++nt) {
#pragma unroll
          for (int e = 0; e < (WIDE ? 4 : 2); ++e) {
            const int key = key0 + nt * 8 + (e & 1);
            const int row = g0 + (e >> 1) * 8;
            const bool ok = key < t_end && key >= t_lo && row < G;
            s[nt][e] = ok ? fmaf(s[nt][e], scale_log2, attn_table_bias_log2(opt, pos - key, kvh * G + row, nh))
                          : -INFINITY;
          }
        }
      } else if (opt.slopes != nullptr) {
        // a bias that grows with the distance, for every row (head) of the tile: its value at
        // this thread's first key of the tile, then a constant step per key; masks only in
        // the last tile (keys beyond the token's own) and the first (keys before the window)
        const int key0 = tile_key0 + 2 * (lane & 3);
        const float at0[2] = {-slope_log2[0] * (float)(pos - key0), -slope_log2[1] * (float)(pos - key0)};
        const bool edge = tile_key0 + DEC_TILE > t_end || tile_key0 < t_lo;
#pragma unroll
        for (int nt = 0; nt < DEC_TILE / 8; ++nt) {
#pragma unroll
          for (int e = 0; e < (WIDE ? 4 : 2); ++e) {
            const float v = fmaf(s[nt][e], scale_log2, fmaf(slope_log2[e >> 1], (float)(nt * 8 + (e & 1)), at0[e >> 1]));
            const int key = key0 + nt * 8 + (e & 1);
            s[nt][e] = (!edge || (key < t_end && key >= t_lo)) ? v : -INFINITY;
          }
        }
      } else if (tile_key0 + DEC_TILE > t_end || tile_key0 < t_lo) {
        // the last tile (keys beyond the token's own) or the first (keys before the window)
        const int key0 = tile_key0 + 2 * (lane & 3);
#pragma unroll
        for (int nt = 0; nt < DEC_TILE / 8; ++nt) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int key = key0 + nt * 8 + (e & 1);
            s[nt][e] = (key < t_end && key >= t_lo) ? s[nt][e] * scale_log2 : -INFINITY;
          }
        }
      } else {
#pragma unroll
        for (int nt = 0; nt < DEC_TILE / 8; ++nt) {
#pragma unroll
          for (int e = 0; e < (WIDE ? 4 : 2); ++e) s[nt][e] *= scale_log2;
        }
      }
      decode_softmax_step<VD, DEC_TILE / 8, WIDE>(s, m, l, o);
      pv_tile<VD, DEC_TILE / 8>(o, s, vt, lane);
      __syncwarp();
      if (++stage == DEC_STAGES) stage = 0;
    }
  };
  if (G > 8) run(std::true_type()); else run(std::false_type());
  cp_async_wait<0>();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
  }

  // merge the block's warps through shared memory (reusing the tile buffers)
  __syncthreads();
  float* red_o = reinterpret_cast<float*>(smem_raw);                 // [warps][16][VD]
  float* red_m = red_o + WARPS * 16 * VD;                        // [warps][16]
  float* red_l = red_m + WARPS * 16;
  float* cta_o = red_l + WARPS * 16;                             // [16][VD] this block's merged partial
  float* cta_ml = cta_o + 16 * VD;                                   // [16][2]
  {
    const int g0 = lane >> 2, c0 = 2 * (lane & 3);
#pragma unroll
    for (int nt = 0; nt < VD / 8; ++nt) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int row = g0 + (e >> 1) * 8, col = nt * 8 + c0 + (e & 1);
        red_o[((size_t)warp * 16 + row) * VD + col] = o[nt][e];
      }
    }
    if ((lane & 3) == 0) {
      red_m[warp * 16 + g0] = m[0];
      red_m[warp * 16 + g0 + 8] = m[1];
      red_l[warp * 16 + g0] = l[0];
      red_l[warp * 16 + g0 + 8] = l[1];
    }
  }
  __syncthreads();
  for (int idx = threadIdx.x; idx < G * vd; idx += WARPS * 32) {
    const int row = idx / vd, d = idx - row * vd;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) M = fmaxf(M, red_m[w * 16 + row]);
    const float m_use = (M == -INFINITY) ? 0.f : M;
    float L = 0.f, acc = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) {
      const float f = exp2f(red_m[w * 16 + row] - m_use);
      L += red_l[w * 16 + row] * f;
      acc += red_o[((size_t)w * 16 + row) * VD + d] * f;
    }
    const int h = kvh * G + row;
    if (n_splits == 1) {
      out[(size_t)seq * out_stride + (size_t)h * vd + d] =
          __float2bfloat16_rn(attn_finish(acc, M, L, opt.sink, attn_gate_factor(opt, seq, h, d, vd) * out_factor,
                                          attn_sink_log2(opt, h)));
    } else if (cluster_merge) {
      // the slices of this (request, KV head) are one thread-block cluster: park the block's
      // partial result in its own shared memory for the merge below
      cta_o[idx] = acc;
      if (d == 0) {
        cta_ml[2 * row] = M;
        cta_ml[2 * row + 1] = L;
      }
    } else {
      const size_t p = ((size_t)seq * nh + h) * n_splits + split;
      part_o[p * vd + d] = acc;
      if (d == 0) {
        part_ml[p * 2] = M;
        part_ml[p * 2 + 1] = L;
      }
    }
  }
  if (n_splits > 1 && cluster_merge) {
    // every block merges its share of the G x VD outputs, reading all slices' partial
    // results (in slice order) from its peers' shared memory
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
    const uint32_t o_addr = (uint32_t)__cvta_generic_to_shared(cta_o);
    const uint32_t ml_addr = (uint32_t)__cvta_generic_to_shared(cta_ml);
    auto peer = [](uint32_t addr, uint32_t rank) {
      uint32_t remote;
      float v;
      asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(addr), "r"(rank));
      asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
      return v;
    };
    const int total = G * vd;
    const int per = (total + n_splits - 1) / n_splits;
    const int e_end = min(total, (split + 1) * per);
    for (int idx = split * per + threadIdx.x; idx < e_end; idx += WARPS * 32) {
      const int row = idx / vd, d = idx - row * vd;
      float ms[8], ls[8], os[8];
#pragma unroll
      for (int sp = 0; sp < 8; ++sp) {
        const bool on = sp < n_splits;
        ms[sp] = on ? peer(ml_addr + (uint32_t)(2 * row) * 4u, sp) : -INFINITY;
        ls[sp] = on ? peer(ml_addr + (uint32_t)(2 * row + 1) * 4u, sp) : 0.f;
        os[sp] = on ? peer(o_addr + (uint32_t)idx * 4u, sp) : 0.f;
      }
      float M = -INFINITY;
#pragma unroll
      for (int sp = 0; sp < 8; ++sp) M = fmaxf(M, ms[sp]);
      float L = 0.f, acc = 0.f;
#pragma unroll
      for (int sp = 0; sp < 8; ++sp) {
        const float f = exp2f(ms[sp] - M);
        L += ls[sp] * f;
        acc += os[sp] * f;
      }
      out[(size_t)seq * out_stride + (size_t)(kvh * G + row) * vd + d] =
          __float2bfloat16_rn(attn_finish(acc, M, L, opt.sink,
                                          attn_gate_factor(opt, seq, kvh * G + row, d, vd) * out_factor,
                                          attn_sink_log2(opt, kvh * G + row)));
    }
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
  }
}

// `vd` values a head; rows of the output `out_stride` apart; a constant factor on it.
__global__ void decode_merge_kernel(__nv_bfloat16* __restrict__ out, const float* __restrict__ part_o,
                                    const float* __restrict__ part_ml, int n_splits, int nh,
                                    AttnOptions opt, int vd, int out_stride, float out_factor) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t row = blockIdx.x;   // seq * nh + head
  const float sink_log2 = attn_sink_log2(opt, (int)(row % nh));
  const float* ml = part_ml + row * n_splits * 2;
  float M = -INFINITY;
  for (int s = 0; s < n_splits; ++s) M = fmaxf(M, ml[2 * s]);
  float L = 0.f;
  for (int s = 0; s < n_splits; ++s) L += ml[2 * s + 1] * exp2f(ml[2 * s] - M);
  for (int d = threadIdx.x; d < vd; d += blockDim.x) {
    float acc = 0.f;
    for (int s = 0; s < n_splits; ++s)
      acc += part_o[(row * n_splits + s) * vd + d] * exp2f(ml[2 * s] - M);
    out[row / nh * (size_t)out_stride + row % nh * vd + d] = __float2bfloat16_rn(attn_finish(acc, M, L, opt.sink,
                                                        attn_gate_factor(opt, row / nh, (int)(row % nh), d, vd) * out_factor,
                                                        sink_log2));
  }
}

template <int HD, int VD, int WARPS>
constexpr size_t decode_smem_bytes() {
  const size_t tiles = (size_t)WARPS * DEC_STAGES * DEC_TILE * (HD + 8 + VD + 8) * sizeof(__nv_bfloat16);
  const size_t red = (size_t)(WARPS * 16 * (VD + 2) + 16 * (VD + 2)) * sizeof(float);
  return tiles > red ? tiles : red;
}

template <int HD, int VD, int WARPS, bool POOLED>
int launch_decode(void* out, float* part_o, float* part_ml, const void* q, int q_stride,
                  const void* k_pages, const void* v_pages, const int* block_table, int bt_stride,
                  const int* positions, int S, int nh, int nkv, int page_size, int window,
                  float scale, int n_splits, const float* rot_cos, const float* rot_sin,
                  int write_cache, AttnOptions opt, QkPrepare prep, PooledKeys pk, cudaStream_t stream) {
  // the new keys and values go into the very pages the kernel reads
  __nv_bfloat16* k_write = write_cache ? (__nv_bfloat16*)const_cast<void*>(k_pages) : nullptr;
  __nv_bfloat16* v_write = write_cache ? (__nv_bfloat16*)const_cast<void*>(v_pages) : nullptr;
  constexpr size_t smem = decode_smem_bytes<HD, VD, WARPS>();
  auto kernel = decode_attention_kernel<HD, VD, WARPS, POOLED>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return HB_LAUNCH_FAILED;
    configured = true;
  }
  dim3 grid(n_splits, nkv, S);
  const int cluster_merge = (n_splits > 1 && n_splits <= 8 && part_o == nullptr) ? 1 : 0;
  if (cluster_merge) {
    // the slices of one (request, KV head) as a cluster: merged through distributed shared memory
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(WARPS * 32);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = n_splits;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = hb_pdl_enabled() ? 2 : 1;
    cudaLaunchKernelEx(&cfg, kernel, (__nv_bfloat16*)out, part_o, part_ml, (const __nv_bfloat16*)q, q_stride,
                       (const __nv_bfloat16*)k_pages, (const __nv_bfloat16*)v_pages, block_table, bt_stride,
                       positions, nh, nkv, page_size, window, scale * LOG2E, n_splits, 1,
                       rot_cos, rot_sin, k_write, v_write, opt, prep, pk);
    return hb_check_launch();
  }
  hb_launch(kernel, dim3(grid), dim3(WARPS * 32), smem, stream, 
      (__nv_bfloat16*)out, part_o, part_ml, (const __nv_bfloat16*)q, q_stride,
      (const __nv_bfloat16*)k_pages, (const __nv_bfloat16*)v_pages, block_table, bt_stride,
      positions, nh, nkv, page_size, window, scale * LOG2E, n_splits, 0,
      rot_cos, rot_sin, k_write, v_write, opt, prep, pk);
  if (n_splits > 1)
    hb_launch(decode_merge_kernel, dim3(S * nh), dim3(VD < 128 ? VD : 128), 0, stream, (__nv_bfloat16*)out, part_o,
              part_ml, n_splits, nh, opt, POOLED ? pk.vd : VD, POOLED ? pk.out_stride : nh * VD,
              POOLED ? pk.factor : 1.f);
  return hb_check_launch();
}

// Clusters of `cluster_size` decode blocks the device keeps resident at once (-1 if the
// query fails): whole clusters are placed inside a GPC, so this can be fewer than the blocks
// that would fit one by one.
template <int HD, int VD, int WARPS, bool POOLED>
int decode_max_clusters(int cluster_size) {
  constexpr size_t smem = decode_smem_bytes<HD, VD, WARPS>();
  auto kernel = decode_attention_kernel<HD, VD, WARPS, POOLED>;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return -1;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(cluster_size, 1, 1);
  cfg.blockDim = dim3(WARPS * 32);
  cfg.dynamicSmemBytes = smem;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cluster_size;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  int n = 0;
  if (cudaOccupancyMaxActiveClusters(&n, kernel, &cfg) != cudaSuccess) return -1;
  return n;
}

}  // namespace
