// Prefill / mixed-batch attention over the paged cache on the 5th-generation tensor
// cores (tcgen05.mma with the score and output tiles in tensor memory), bfloat16,
// head sizes 64 and 128.
//
// A block takes one KV head and up to 128 query rows = floor(128/G) consecutive tokens of one
// request times the G query heads that share the KV head (the last rows idle when G does
// not divide 128), and walks the keys the rows may see in
// tiles of 128:
//     TMA        pages of K and V (boxes of page_size x 64 elements, 128-byte swizzle)
//                -> a two-stage ring in shared memory
//     MMA 1      S[128 x 128] = Q K^T           (Q staged once, K-major; K tile K-major)
//     softmax    8 warps, two threads per row: scale, mask by position (causal, window),
//                maximum and sum in float32, P = exp2(.) as bfloat16 into shared
//                memory in the operand layout
//     MMA 2      O[128 x hd] += P V             (V tile as an MN-major operand); the output
//                accumulates in tensor memory over all key tiles, relative to a reference
//                maximum per row that the softmax warps move (rescaling output and sum) only
//                when the true maximum has run ahead of it by more than 2^8; they read the
//                output back once, at the end, and divide by the sum.
// Formulas: python/helios/exec/paged_attn.py:368-408 (scores * scale, key position > query
// position masked, softmax in float32, times V), head mapping :248-261.
//
// Every mbarrier wait is bounded; on a timeout the block raises the error word, frees its
// tensor memory and returns.
//
// Compiled by attention_tc.cu (values of the keys' size, every option) and attention_tc_pooled.cu
// (POOLED: values of a size of their own, means of whole blocks behind the window as tiles of
// their own ahead of the window's, head sizes that are any multiple of 8: the copies fill the
// columns beyond them with zeros).
#pragma once
#include "tcgen05.cuh"
#include "attention_options.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;
constexpr int TILE = 128;            // query rows and keys per tile
constexpr int TC_THREADS = 352;      // warp 0: TMA of K, warp 1: MMA, warps 2-9: softmax, warp 10: TMA of V
constexpr int SOFTMAX_THREADS = 256;

// Means of whole blocks of `pool` tokens behind the window, a key and a value each in pages of
// their own; block b is seen at position p if (b + 1) * pool <= p - window + 1.
struct PooledTiles {
  const int* table;         // [requests, table_stride]
  int table_stride;
  int pool;                 // 0: none
  int hd, vd;               // sizes (multiples of 8) at most the ones the kernel is compiled for
  int out_stride;           // elements between rows of the output
  float factor;             // a constant on the output
  int side_by_side;         // a token's heads lie beside each other in ONE row of the maps (no page a head):
                            // head h's columns begin at h * hd / h * vd, a page is page_size rows
};

struct AttnArgs {
  AttnOptions opt;          // distance bias, sink, gate (all off when zeroed)
  const float* bias_t;      // the bias table by distance TRANSPOSED, [heads, opt.bias_rows] (or null): a
                            // warp's rows are few heads x consecutive tokens, so its look-ups for one
                            // key fall into a few short runs of one head's row
  __nv_bfloat16* out;
  const __nv_bfloat16* q;
  int q_stride;
  const int* block_table;
  int bt_stride;
  const int* q_tiles;       // (request, first local token) per tile
  const int* cu_tokens;
  const int* start_pos;
  int nh, nkv, page_size, window;
  float scale_log2;
  int* error;
};

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void named_barrier(int id, int threads) {
  asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory");
}
__device__ __forceinline__ void st_shared_v4(uint32_t addr, uint32_t a, uint32_t b, uint32_t c, uint32_t d) {
  asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(addr), "r"(a), "r"(b), "r"(c), "r"(d) : "memory");
}
// byte offset of 16-byte chunk `c8` (0..7) of row `row` in a [rows x 128 bytes] tile with
// the 128-byte swizzle (chunk index XOR row mod 8)
__device__ __forceinline__ uint32_t swz(int row, int c8) {
  return (uint32_t)((row >> 3) * 1024 + (row & 7) * 128 + ((c8 ^ (row & 7)) << 4));
}

// Stages of the K and the V ring that fit beside Q and P in 227 KB.
template <int HD, int VD> struct TcStages {
  static constexpr int UNITS = 11;                  // blocks of 16 KB for Q, K and V
  static constexpr int KH = HD / 64, VH = VD / 64;
  static constexpr int K = KH + 2 * KH + VH <= UNITS ? 2 : 1;
  static constexpr int V = KH + K * KH + 2 * VH <= UNITS ? 2 : 1;
  static_assert(KH + K * KH + V * VH <= UNITS, "Q, K, V and P do not fit shared memory");
  static constexpr size_t BYTES = (size_t)(KH + K * KH + V * VH + 2) * TILE * 128 + 1024 + 4096;
};

template <int HD, int VD, bool POOLED>
__global__ void __launch_bounds__(TC_THREADS, 1)
attention_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                            const __grid_constant__ CUtensorMap map_pk, const __grid_constant__ CUtensorMap map_pv,
                            AttnArgs a, PooledTiles pl) {
  static_assert(POOLED || HD == VD, "values of another size come with the pooled kernels");
  constexpr int KH = HD / 64, VH = VD / 64;         // 64-element halves of the head dimensions
  constexpr int KST = TcStages<HD, VD>::K, VST = TcStages<HD, VD>::V;
  constexpr int HALF_BYTES = TILE * 128;            // one [128 rows x 64 elements] block
  constexpr int QK_BYTES = KH * HALF_BYTES;         // a Q or K tile
  constexpr int V_BYTES = VH * HALF_BYTES;
  constexpr int P_BYTES = 2 * HALF_BYTES;           // 128 rows x 128 keys
  constexpr uint32_t TMEM_COLS = VD > 128 ? 512 : 256;
  constexpr uint32_t S_COL = 0, O_COL = 128;

  extern __shared__ unsigned char smem_raw[];
  pdl_launch_dependents();
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  unsigned char* aligned = smem_raw + (base - smem_u32(smem_raw));
  const uint32_t q_smem = base;
  const uint32_t k_smem = q_smem + QK_BYTES;                // KST stages
  const uint32_t v_smem = k_smem + KST * QK_BYTES;          // VST stages
  const uint32_t p_smem = v_smem + VST * V_BYTES;
  uint64_t* bars = reinterpret_cast<uint64_t*>(aligned + (1 + KST) * QK_BYTES + VST * V_BYTES + P_BYTES);
  // 0,1: K full; 2,3: K empty; 4: q ready; 5: s full; 6: p ready; 7: o full; 8: s free;
  // 9,10: V full; 11,12: V empty
  float* l_exchange = reinterpret_cast<float*>(bars + 14);  // [128]
  float* max_exchange = l_exchange + TILE;                  // [2 tiles][2 halves][128]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(max_exchange + 4 * TILE);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  auto bar = [&](int i) { return smem_u32(bars + i); };

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int G = a.nh / a.nkv;
  const int TQ = TILE / G;                            // tokens per tile
  // KV heads fastest: the tiles come longest first, and so do the blocks, whatever the head
  const int kvh = blockIdx.x % a.nkv, q_tile = blockIdx.x / a.nkv;
  const int seq = a.q_tiles[2 * q_tile], t0 = a.q_tiles[2 * q_tile + 1];

  if (threadIdx.x == 0) {
    mbar_init(bar(0), 1); mbar_init(bar(1), 1);
    mbar_init(bar(2), 1); mbar_init(bar(3), 1);
    mbar_init(bar(4), SOFTMAX_THREADS / 32);     // one arrival per softmax warp
    mbar_init(bar(5), 1);
    mbar_init(bar(6), SOFTMAX_THREADS / 32);
    mbar_init(bar(7), 1);
    mbar_init(bar(8), SOFTMAX_THREADS / 32);
    mbar_init(bar(9), 1); mbar_init(bar(10), 1);
    mbar_init(bar(11), 1); mbar_init(bar(12), 1);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  pdl_wait();     // everything below reads what earlier kernels wrote
  const int tok0 = a.cu_tokens[seq], n_tok = a.cu_tokens[seq + 1] - tok0;
  const int sp = a.start_pos[seq];
  const int p_first = sp + t0;
  const int p_last = sp + min(n_tok, t0 + TQ) - 1;
  const int k_min = (a.window > 0 && p_first - a.window + 1 > 0) ? p_first - a.window + 1 : 0;
  const int kt_begin = k_min / TILE, kt_end = p_last / TILE + 1;
  // The first keys a window keeps come as tiles of their own BEFORE the window's: iteration
  // it < kept_tiles walks tile it, the others the tiles from kt_begin on.
  const int keep = a.window > 0 ? a.opt.keep_first : 0;
  const int kept_tiles = min((min(keep, k_min) + TILE - 1) / TILE, kt_begin);
  // With POOLED the blocks behind the window take that place: tiles of 128 blocks, up to the last
  // block some row sees.
  auto blocks_seen = [&](int p) { return POOLED && pl.pool > 0 && p - a.window + 1 > 0 ? (p - a.window + 1) / pl.pool : 0; };
  const int blocks_last = blocks_seen(p_last);
  const int pre_tiles = POOLED ? (blocks_last + TILE - 1) / TILE : kept_tiles;
  auto tile_of = [&](int it) { return it < pre_tiles ? it : kt_begin + it - pre_tiles; };
  // a tile beyond the request's tokens (padding of a captured step's tile list) has no work
  const int n_it = t0 < n_tok ? pre_tiles + kt_end - kt_begin : 0;
  const int* table = a.block_table + (size_t)seq * a.bt_stride;
  const int ps = a.page_size;
  const int pages_per_tile = TILE / ps;

  if (warp == 0 || warp == 10) {
    // ---------------------------------------------------------------- TMA producers
    // Warp 0 copies the K tiles, warp 10 the V tiles, each through a ring of two stages of
    // its own: a K stage is free again as soon as the scores of its tile are computed, long
    // before its V stage, so the next keys arrive while the softmax of this tile still runs.
    // Lane i looks up and copies page i of the tile (the look-ups of a tile's pages would
    // otherwise wait for one another); lane 0 waits for the stage and announces the bytes.
    {
      const bool is_v = warp == 10;
      const uint32_t ring = is_v ? v_smem : k_smem;
      const int full0 = is_v ? 9 : 0, empty0 = is_v ? 11 : 2;
      const int stages = is_v ? VST : KST, halves = is_v ? VH : KH, tile_bytes = is_v ? V_BYTES : QK_BYTES;
      for (int it = 0; it < n_it; ++it) {
        const int s = it % stages;
        const int key_base = tile_of(it) * TILE;
        const bool blocks = POOLED && it < pre_tiles;
        const CUtensorMap* map = blocks ? (is_v ? &map_pv : &map_pk) : (is_v ? &map_v : &map_k);
        const int* tab = blocks ? pl.table + (size_t)seq * pl.table_stride : table;
        // pages that hold at least one key some row may see: inside the first row's window
        // or among the kept first keys (pages in between may have been given back)
        const int key0 = key_base + lane * ps;
        const bool mine = lane < pages_per_tile &&
                          (blocks ? key0 < blocks_last : (key0 + ps - 1 >= k_min || key0 < keep) && key0 <= p_last);
        const int count = __popc(__ballot_sync(0xffffffffu, mine));
        int row = 0;
        const bool wide = POOLED && pl.side_by_side;
        const int col = wide ? kvh * (is_v ? pl.vd : pl.hd) : 0;
        if (mine) {                                                                 // before the wait
          const int page = tab[(key_base + lane * ps) / ps];
          row = wide ? page * ps : (page * a.nkv + kvh) * ps;
        }
        int go = 1;
        if (lane == 0) {
          go = mbar_wait(bar(empty0 + s), ((it / stages) & 1) ^ 1, abort_flag, a.error, 11) ? 1 : 0;
          if (go) mbar_expect_tx(bar(full0 + s), (uint32_t)(count * ps * 128 * halves));
        }
        go = __shfl_sync(0xffffffffu, go, 0);
        if (!go) break;
        if (mine) {
          const uint32_t off = (uint32_t)(lane * ps * 128);
#pragma unroll
          for (int hh = 0; hh < (KH > VH ? KH : VH); ++hh)
            if (hh < halves)
              tma_load_2d(ring + s * tile_bytes + hh * HALF_BYTES + off, map, bar(full0 + s), col + hh * 64, row);
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      // ------------------------------------------------------------ MMA issuer
      constexpr uint32_t idesc_qk = instr_desc(TILE, TILE);
      constexpr uint32_t idesc_pv = instr_desc_b_mn(TILE, VD);
      // S(i+1) = Q K(i+1)^T is issued as soon as the softmax warps have taken S(i) into
      // registers, so that it runs under their exponentials; O_tile(i) = P(i) V(i) follows
      // when P(i) is written.
      bool ok = mbar_wait(bar(4), 0, abort_flag, a.error, 12);
      auto issue_qk = [&](int it) {
        const int s = it % KST;
        if (!mbar_wait(bar(s), (it / KST) & 1, abort_flag, a.error, 13)) return false;
        tc_fence_after();
        const uint32_t ks = k_smem + s * QK_BYTES;
#pragma unroll
        for (int hh = 0; hh < KH; ++hh)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16(tmem_base + S_COL, smem_desc(q_smem + hh * HALF_BYTES + k * 32),
                      smem_desc(ks + hh * HALF_BYTES + k * 32), idesc_qk, (hh | k) ? 1u : 0u);
        umma_commit(bar(2 + s));      // the K stage is free once the scores are there
        umma_commit(bar(5));
        return true;
      };
      if (ok && n_it > 0) ok = issue_qk(0);
      for (int it = 0; it < n_it && ok; ++it) {
        const int s = it % VST;
        if (it + 1 < n_it) {
          ok = mbar_wait(bar(8), it & 1, abort_flag, a.error, 17);     // S(it) is in registers
          if (!ok) break;
          tc_fence_after();
          ok = issue_qk(it + 1);
          if (!ok) break;
        }
        ok = mbar_wait(bar(9 + s), (it / VST) & 1, abort_flag, a.error, 18);     // V(it) has arrived
        if (!ok) break;
        ok = mbar_wait(bar(6), it & 1, abort_flag, a.error, 14);
        if (!ok) break;
        tc_fence_after();
        const uint32_t vs = v_smem + s * V_BYTES;
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          umma_bf16(tmem_base + O_COL, smem_desc(p_smem + (kk >> 2) * HALF_BYTES + (kk & 3) * 32),
                    smem_desc_mn(vs + kk * 2048, HALF_BYTES, 1024), idesc_pv, (it | kk) ? 1u : 0u);
        umma_commit(bar(11 + s));    // the V stage is free
        umma_commit(bar(7));         // O_tile complete
      }
    }
    __syncwarp();
  } else {
    // -------------------------------------------------------------- softmax warps
    const int sw = warp - 2;                       // 0..7 (warps 2..9)
    const int quarter = warp & 3;                  // lanes of tensor memory this warp may read
    const int half = sw >> 2;                      // which 64 keys / which half of hd this thread owns
    const int m = quarter * 32 + lane;             // row of the tile
    const int tl = t0 + m / G, g = m % G;
    const bool row_valid = m < TQ * G && tl < n_tok;       // rows beyond TQ * G idle when G does not divide 128
    const int pr = sp + tl;                        // the row's position
    const int tid = threadIdx.x - 64;
    // with a distance bias the scores are scaled and biased as they come out of tensor
    // memory, and the factor on them further down is 1
    const bool biased = a.opt.slopes != nullptr;
    const bool tabled = a.bias_t != nullptr;
    const float slope_log2 = (biased && row_valid) ? a.opt.slopes[kvh * G + g] * LOG2E : 0.f;
    const float sc = (biased || tabled) ? 1.f : a.scale_log2;
    const float* bias_row = tabled ? a.bias_t + (size_t)(row_valid ? kvh * G + g : 0) * a.opt.bias_rows : nullptr;

    // stage Q: rows = (token, head) pairs, swizzled K-major; invalid rows are zero.  All
    // loads of a thread are issued before the first store (one round trip, not one each).
    {
      constexpr int PER_THREAD = TILE * (HD / 8) / SOFTMAX_THREADS;
      uint4 qv[PER_THREAD];
#pragma unroll
      for (int i = 0; i < PER_THREAD; ++i) {
        const int idx = tid + i * SOFTMAX_THREADS;
        const int row = idx / (HD / 8), c = idx - row * (HD / 8);
        const int rt = t0 + row / G, rg = row % G;
        qv[i] = make_uint4(0, 0, 0, 0);
        const int hd = POOLED ? pl.hd : HD;
        if (row < TQ * G && rt < n_tok && c * 8 < hd)
          qv[i] = *reinterpret_cast<const uint4*>(a.q + (size_t)(tok0 + rt) * a.q_stride +
                                                  (size_t)(kvh * G + rg) * hd + c * 8);
      }
#pragma unroll
      for (int i = 0; i < PER_THREAD; ++i) {
        const int idx = tid + i * SOFTMAX_THREADS;
        const int row = idx / (HD / 8), c = idx - row * (HD / 8);
        st_shared_v4(q_smem + (c >> 3) * HALF_BYTES + swz(row, c & 7), qv[i].x, qv[i].y, qv[i].z, qv[i].w);
      }
    }
    fence_async_smem();
    __syncwarp();
    if (lane == 0) mbar_arrive(bar(4));

    constexpr int OWN = VD / 2;                    // output columns this thread rescales and writes
    // The output accumulates in tensor memory over all key tiles, relative to a reference
    // maximum m_ref per row that is only moved when the true maximum has run ahead of it by
    // more than LAG (then the output and the sum are rescaled); exponentials are at most
    // 2^LAG meanwhile, and the final quotient does not depend on the reference.
    constexpr float LAG = 8.f;
    float m_ref = -INFINITY, l_run = 0.f;
    const uint32_t lane_addr = tmem_base + ((uint32_t)(quarter * 32) << 16);
    bool ok = true;
    for (int it = 0; it < n_it; ++it) {
      const int key_base = tile_of(it) * TILE;
      if (!mbar_wait(bar(5), it & 1, abort_flag, a.error, 15)) { ok = false; break; }
      tc_fence_after();
      const bool blocks = POOLED && it < pre_tiles;
      const bool masked_tile = blocks ? key_base + TILE > blocks_seen(p_first)
                                      : key_base + TILE - 1 > p_first || key_base < k_min ||
                                        (a.window > 0 && key_base <= p_last - a.window);
      // this thread's 64 scores stay in registers; the maximum goes over to the other
      // thread of the row through shared memory
      float sv[64];
      {
        float v0[32], v1[32];
        tmem_ld32(lane_addr + S_COL + half * 64, v0);
        tmem_ld32(lane_addr + S_COL + half * 64 + 32, v1);
#pragma unroll
        for (int j = 0; j < 32; ++j) { sv[j] = v0[j]; sv[32 + j] = v1[j]; }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar(8));        // the score tile may be overwritten
      if (biased) {
        const float at0 = slope_log2 * (float)(key_base + half * 64 - pr);      // the bias at this thread's first key
#pragma unroll
        for (int j = 0; j < 64; ++j) sv[j] = fmaf(sv[j], a.scale_log2, fmaf(slope_log2, (float)j, at0));
      }
      if (tabled) {
        // the bias of every score by its distance; beyond the table's last row that row's
        const int d0 = pr - (key_base + half * 64), last = a.opt.bias_rows - 1;
#pragma unroll
        for (int j = 0; j < 64; ++j) {
          const int d = d0 - j;
          const float b = __ldg(bias_row + (d < 0 ? 0 : (d < last ? d : last)));
          sv[j] = fmaf(b, LOG2E, sv[j] * a.scale_log2);
        }
      }
      if (masked_tile) {
        // columns of this thread's 64 keys the row may see: [lo, hi]
        const int col0 = key_base + half * 64;
        const int hi = (blocks ? blocks_seen(pr) - 1 : pr) - col0;
        const int lo = (a.window > 0 && !blocks ? pr - a.window + 1 : 0) - col0;
#pragma unroll
        for (int j = 0; j < 64; ++j)
          if ((j < lo && col0 + j >= keep) || j > hi) sv[j] = -INFINITY;
      }
      float mx4[4] = {sv[0], sv[1], sv[2], sv[3]};
#pragma unroll
      for (int j = 4; j < 64; ++j) mx4[j & 3] = fmaxf(mx4[j & 3], sv[j]);
      float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      max_exchange[((it & 1) * 2 + half) * TILE + m] = mx;
      named_barrier(2 + quarter, 64);
      mx = fmaxf(mx, max_exchange[((it & 1) * 2 + (half ^ 1)) * TILE + m]) * sc;
      // move the reference?  Both threads of a row see the same numbers; the rows of a warp
      // decide together, because tensor memory is read and written by whole warps.
      const bool move = mx > m_ref + LAG || (m_ref == -INFINITY && mx > -INFINITY);
      const bool rescale = __any_sync(0xffffffffu, move) && it > 0;
      float factor = 1.f;
      if (move) {
        factor = fast_exp2(m_ref - mx);          // 0 while nothing has been added yet
        m_ref = mx;
        l_run *= factor;
      }
      const float m_use = (m_ref == -INFINITY) ? 0.f : m_ref;
      // the exponentials of this tile, packed, wait in registers: the product of the tile
      // before, which still reads P, finishes under this work
      float sum4[4] = {0.f, 0.f, 0.f, 0.f};
      uint32_t packed[32];
#pragma unroll
      for (int j = 0; j < 32; ++j) {
        const float p0 = fast_exp2(fmaf(sv[2 * j], sc, -m_use));
        const float p1 = fast_exp2(fmaf(sv[2 * j + 1], sc, -m_use));
        sum4[j & 3] += p0 + p1;
        __nv_bfloat162 pk = __floats2bfloat162_rn(p0, p1);
        packed[j] = *reinterpret_cast<uint32_t*>(&pk);
      }
      l_run += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
      if (it > 0) {
        // P of the tile before has been read, and its product is in the output
        if (!mbar_wait(bar(7), (it - 1) & 1, abort_flag, a.error, 16)) { ok = false; break; }
        tc_fence_after();
        if (rescale) {
#pragma unroll
          for (int c = 0; c < OWN / 32; ++c) {
            float v[32];
            tmem_ld32(lane_addr + O_COL + half * OWN + c * 32, v);
#pragma unroll
            for (int j = 0; j < 32; ++j) v[j] *= factor;
            tmem_st32(lane_addr + O_COL + half * OWN + c * 32, v);
          }
        }
      }
#pragma unroll
      for (int c8 = 0; c8 < 8; ++c8)
        st_shared_v4(p_smem + half * HALF_BYTES + swz(m, c8), packed[4 * c8], packed[4 * c8 + 1],
                     packed[4 * c8 + 2], packed[4 * c8 + 3]);
      // V rows of keys past the last position (unwritten slots, pages that were not copied)
      // must not be NaN or Inf when they meet their zero probabilities
      {
        const int s = it % VST;
        auto zero_rows = [&](int row_begin, int row_end) {
          for (int idx = tid + row_begin * VH * 8; idx < row_end * VH * 8; idx += SOFTMAX_THREADS) {
            const int row = idx / (VH * 8), rest = idx - row * (VH * 8);
            st_shared_v4(v_smem + s * V_BYTES + (rest >> 3) * HALF_BYTES + row * 128 + (rest & 7) * 16,
                         0, 0, 0, 0);
          }
        };
        if (blocks) {
          if (key_base + TILE > blocks_last) {
            if (!mbar_wait(bar(9 + s), (it / VST) & 1, abort_flag, a.error, 19)) { ok = false; break; }
            zero_rows(blocks_last - key_base, TILE);
          }
        } else if (key_base + TILE - 1 > p_last || key_base < k_min) {
          // the copies of this V tile must have landed first: they bring whole pages
          if (!mbar_wait(bar(9 + s), (it / VST) & 1, abort_flag, a.error, 19)) { ok = false; break; }
          if (key_base + TILE - 1 > p_last) zero_rows(p_last + 1 - key_base, TILE);
          // pages wholly before the window of the first row (and behind the kept first keys)
          // were not copied either
          if (key_base < k_min) {
            const int z0 = keep > key_base ? min(TILE, ((keep - key_base + ps - 1) / ps) * ps) : 0;
            const int z1 = min(TILE, ((k_min - key_base) / ps) * ps);
            if (z1 > z0) zero_rows(z0, z1);
          }
        }
      }
      tc_fence_before();
      fence_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar(6));
    }
    const bool have = ok && n_it > 0 && mbar_wait(bar(7), (n_it - 1) & 1, abort_flag, a.error, 16);
    if (have) tc_fence_after();

    // the two threads of a row add their sums
    if (half == 1) l_exchange[m] = l_run;
    named_barrier(1, SOFTMAX_THREADS);
    if (half == 0) {
      const float other = l_exchange[m];
      l_exchange[m] = l_run;
      l_run += other;
    }
    named_barrier(1, SOFTMAX_THREADS);
    if (half == 1) l_run += l_exchange[m];
    // the output leaves tensor memory 32 columns at a time: 1 / sum, gate, bfloat16
    const bool store = row_valid && !*abort_flag;
    const int h = kvh * G + g;
    const int vd = POOLED ? pl.vd : VD;
    // the factor on every value of the row: 1 / l_run without a sink or a gate
    const float inv = have && store ? attn_finish(1.f, m_ref, l_run, a.opt.sink,
                                                  (a.opt.gate_wide ? 1.f : attn_gate_factor(a.opt, tok0 + tl, h)) *
                                                      (POOLED ? pl.factor : 1.f),
                                                  attn_sink_log2(a.opt, h))
                                    : 0.f;
    __nv_bfloat16* dst = a.out + (size_t)(tok0 + tl) * (POOLED ? pl.out_stride : a.nh * HD) + (size_t)h * vd + half * OWN;
    const __nv_bfloat16* grow = a.opt.gate != nullptr && a.opt.gate_wide
        ? a.opt.gate + (size_t)(tok0 + tl) * a.opt.gate_stride + (size_t)h * vd + half * OWN : nullptr;
    const bool gate_vec = (reinterpret_cast<uintptr_t>(grow) & 15) == 0;
#pragma unroll
    for (int c = 0; c < OWN / 32; ++c) {
      if (!have) break;
      float v[32];
      tmem_ld32(lane_addr + O_COL + half * OWN + c * 32, v);
      if (!store) continue;
      if (grow != nullptr) {
        // a gate per output value: eight at a time where the row allows 16-byte loads
#pragma unroll
        for (int j = 0; j < 32; j += 8) {
          if (gate_vec) {
            const uint4 gv = *reinterpret_cast<const uint4*>(grow + c * 32 + j);
            const uint32_t gw[4] = {gv.x, gv.y, gv.z, gv.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 gf = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gw[e]));
              v[j + 2 * e] *= 1.f / (1.f + __expf(-gf.x));
              v[j + 2 * e + 1] *= 1.f / (1.f + __expf(-gf.y));
            }
          } else {
#pragma unroll
            for (int e = 0; e < 8; ++e) v[j + e] *= attn_gate_factor(a.opt, tok0 + tl, h, half * OWN + c * 32 + j + e, vd);
          }
        }
      }
#pragma unroll
      for (int j = 0; j < 32; j += 8) {
        if (POOLED && half * OWN + c * 32 + j >= vd) break;
        uint32_t w[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          __nv_bfloat162 pk = __floats2bfloat162_rn(v[j + 2 * e] * inv, v[j + 2 * e + 1] * inv);
          w[e] = *reinterpret_cast<uint32_t*>(&pk);
        }
        *reinterpret_cast<uint4*>(dst + c * 32 + j) = make_uint4(w[0], w[1], w[2], w[3]);
      }
    }
    if (have) tc_fence_before();
  }

  tc_fence_before();
  __syncthreads();
  if (*abort_flag && threadIdx.x == 0) {
    for (int i = 0; i < 2000; ++i) __nanosleep(100);
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
}

}  // namespace
