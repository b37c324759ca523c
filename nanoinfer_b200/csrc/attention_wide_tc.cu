// Attention for prompt portions on the fifth-generation tensor cores where a cached row is wider than one swizzle row of 64
// values (bfloat16), in two shapes of the cache:
//
//   keys and values in planes of their own, rows of row_dim values (up to 256).  A head may own a part of the key row only:
//   with `maps` > 1 query head h scores against the values [m map_dim, (m + 1) map_dim) of its key/value head's row,
//   m = h % maps (differential attention lays the keys of a head's maps side by side; the query is zero elsewhere, so the
//   bounds need not fall on a boundary of anything), and v_cols of the value row count;
//
//   one plane whose row is key and value at once (a latent [c | k_rot] shared by all heads, latent_attention.cu; rows up to
//   320, v_cols = kv_rank up to 256): a tile is loaded once and read as both.
//
// One block takes 128 consecutive query rows of one request and one head and walks the keys in tiles of 64:
//   warp 0      the producer: Q once; then a tile at a time, 16 rows x 64 values a TMA load (a lane each, with its own look-up
//               in the block table), into a ring of stages of 128-byte-swizzled shared memory: chunks of [64 keys][64 values],
//               those of the key row that the head needs, then those of the value row;
//   warp 1      the MMAs: S = Q K^T (128 x 64 x the head's part of the row) into one of two score buffers in tensor memory;
//               O += P V (128 x v_cols x 64) with P from shared memory and V as it lies, keys down the rows, an MN-major
//               operand of chunks side by side, accumulated in tensor memory over all tiles.  Whatever is ready goes next,
//               P V first (it frees a stage);
//   warps 2..5  the softmax, a thread a row: scores times log2(e) (capped first where asked for), running maximum raised only
//               when a tile exceeds it by more than 2^8 (O is then scaled in tensor memory), P as bfloat16, the sum in
//               32-bit; at the end an optional learned sink, the division, an optional sigmoid gate per row and head or per
//               element, and the store (bfloat16, or 32-bit floats).
// Ahead of the window's tiles come those of pooled blocks where there are any: rows of another list of pages of the same
// cache, one key and value for `pool` positions that lie wholly behind the window; every row knows how many it sees.
// Keys outside [lowest visible, last row] are masked; their rows are read from the nearest unit of the request that is
// there.  What a box reaches beyond the row, or beyond the step's rows, reads as zeros.
//
// Every wait on a barrier is bounded: a wait that runs out sets the block's abort flag and the device status word, every
// role leaves its loop, tensor memory is freed, and the kernel returns.
#include "api.h"
#include "attention_extras.cuh"
#include "common.cuh"
#include "tcgen05.cuh"

namespace nib {

constexpr int LP_BM = 128, LP_BN = 64, LP_UNIT = 16, LP_THREADS = 192, LP_NBUF = 2, LP_MAX_STAGES = 4;
constexpr int LP_MAX_SLOTS = 8, LP_MAX_V_CHUNKS = 4;          // chunks of a stage (four lanes each), values <= 256
constexpr int LP_CHUNK_Q = LP_BM * 128, LP_CHUNK_K = LP_BN * 128, LP_P_BYTES = LP_BM * 128;
constexpr uint32_t LP_O_COL = LP_NBUF * LP_BN, LP_TMEM_COLS = 512;
constexpr float LP_RAISE = 8.0f;

struct LpParams {
  const int* block_table;
  int max_blocks;
  const int* tiles;            // pairs (entry, first row within the entry), 128 rows each
  const int* entry_start;
  const int* entry_pos0;
  int page_size, n_pages, n_head, n_kv_head, planes;
  int row_dim, maps, map_dim;   // a head's keys: values (h % maps) * map_dim .. + map_dim of the row
  int v_cols, v_chunks;         // values of the result, chunks of the value row
  int k_slots, stages;          // chunks of keys a stage holds room for
  float scale, softcap;
  int window;
  const float* gate;
  int ldg, gate_dim;            // gate_dim 0: one gate a head, else one for each of a head's first gate_dim values
  const float* sinks;           // a logit per head that joins the denominator (null: none)
  int pool;                     // > 0: blocks of so many positions behind the window are one key and value each,
  const int* pool_table;        // rows of these pages
  void* out;
  int ldo, out_head, out32;     // rows and heads of the result, in elements
  int* status;
};

__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* map, uint64_t* bar, int x, int y, int z) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
      ::"r"(smem_u32(dst)), "l"((uint64_t)map), "r"(smem_u32(bar)), "r"(x), "r"(y), "r"(z)
      : "memory");
}
__device__ __forceinline__ float lp_pow2(float x) {   // the hardware's 2^x (relative error about 2^-22; 2^-inf = 0)
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float lp_sigmoid(float x) { return 1.0f / (1.0f + __expf(-x)); }
__device__ __forceinline__ void lp_tmem_ld32(uint32_t taddr, float* v) {
  uint32_t r[32];
  tmem_ld16_issue(taddr, r);
  tmem_ld16_issue(taddr + 16, r + 16);
  tmem_ld_wait();
#pragma unroll
  for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(r[i]);
}
__device__ __forceinline__ void lp_tmem_st16(uint32_t taddr, const float* v) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
      ::"r"(taddr), "r"(__float_as_uint(v[0])), "r"(__float_as_uint(v[1])), "r"(__float_as_uint(v[2])),
        "r"(__float_as_uint(v[3])), "r"(__float_as_uint(v[4])), "r"(__float_as_uint(v[5])), "r"(__float_as_uint(v[6])),
        "r"(__float_as_uint(v[7])), "r"(__float_as_uint(v[8])), "r"(__float_as_uint(v[9])), "r"(__float_as_uint(v[10])),
        "r"(__float_as_uint(v[11])), "r"(__float_as_uint(v[12])), "r"(__float_as_uint(v[13])), "r"(__float_as_uint(v[14])),
        "r"(__float_as_uint(v[15]))
      : "memory");
}

__device__ __forceinline__ bool lp_test(uint64_t* bar, uint32_t parity) {   // has the phase completed?  (does not wait)
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred P1;\n\t"
      "mbarrier.test_wait.parity.shared::cta.b64 P1, [%1], %2;\n\t"
      "selp.b32 %0, 1, 0, P1;\n\t}"
      : "=r"(ok)
      : "r"(smem_u32(bar)), "r"(parity)
      : "memory");
  return ok != 0;
}

__global__ void __launch_bounds__(LP_THREADS, 1)
attention_wide_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv,
                         const LpParams prm) {
  extern __shared__ uint8_t lp_smem_raw[];
  // tiles must start on a 1024-byte boundary for the 128-byte swizzle
  uint8_t* smem = reinterpret_cast<uint8_t*>(((uintptr_t)lp_smem_raw + 1023) & ~(uintptr_t)1023);
  const bool shared_row = prm.planes == 1;              // one row is key and value
  const int h = blockIdx.x, hk = h / (prm.n_head / prm.n_kv_head);
  // the head's part of the key row: steps of 16 values, chunks of 64
  const int k_from = (h % prm.maps) * prm.map_dim, ks_lo = k_from / 16, ks_hi = (k_from + prm.map_dim + 15) / 16;
  const int c_lo = ks_lo / 4, nk = (ks_hi + 3) / 4 - c_lo;
  const int nv = prm.v_chunks, stages = prm.stages;
  const int n_slots = prm.k_slots + (shared_row ? 0 : nv);              // of a stage
  const int stage_bytes = n_slots * LP_CHUNK_K, v_off = shared_row ? 0 : prm.k_slots * LP_CHUNK_K;
  uint8_t* q_s = smem;                                  // [chunks][128 rows][64]
  uint8_t* k_s = q_s + prm.k_slots * LP_CHUNK_Q;        // [stages][key chunks, value chunks][64 keys][64]
  uint8_t* p_s = k_s + stages * stage_bytes;            // [2][128 rows][64 keys]
  __shared__ __align__(8) uint64_t q_full, k_full[LP_MAX_STAGES], k_empty[LP_MAX_STAGES], s_full[LP_NBUF], p_full[LP_NBUF],
      o_full[LP_NBUF];
  __shared__ uint32_t tmem_base_sh;
  __shared__ int abort_sh;
  volatile int* abort_flag = &abort_sh;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // (heads are the fast index of the grid: blocks start in the order of the tile list, longest first)
  const int e = prm.tiles[2 * blockIdx.y], q_off = prm.tiles[2 * blockIdx.y + 1];
  const int row0 = prm.entry_start[e] + q_off;                    // first row of the tile in the step
  const int n_rows = min(LP_BM, prm.entry_start[e + 1] - row0);
  const int pos_first = prm.entry_pos0[e] + q_off;                // position of the tile's first row
  const int pos_last = pos_first + n_rows - 1;
  const int* table = prm.block_table + (size_t)e * prm.max_blocks;
  const int window = prm.window;
  const int key_lo = (window > 0 && pos_first - window + 1 > 0) ? pos_first - window + 1 : 0;
  // the pooled blocks that the tile's rows see come first, in tiles of their own
  const int nb_last = pooled_blocks_seen(pos_last, window, prm.pool), n_pool = (nb_last + LP_BN - 1) / LP_BN;
  const int* pool_table = prm.pool_table + (size_t)e * prm.max_blocks;
  const int tile_first = key_lo / LP_BN - n_pool, n_it = pos_last / LP_BN - tile_first + 1;

  if (threadIdx.x == 0) {
    abort_sh = 0;
    mbar_init(&q_full, 1);
    for (int i = 0; i < LP_MAX_STAGES; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
    }
    for (int i = 0; i < LP_NBUF; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&p_full[i], 128);
      mbar_init(&o_full[i], 1);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  pdl_wait();   // the queries, and this step's rows of the cache, come from the kernels ahead
  // Tensor memory is taken once the kernels ahead, which may hold some, are done, and the kernels behind, which may want
  // some, are let go only when it has been taken: no block waits for memory that is held by one that waits for it.
  if (warp == 1) tmem_alloc(&tmem_base_sh, LP_TMEM_COLS);
  tc_fence_before();
  __syncthreads();
  pdl_trigger();
  tc_fence_after();
  const uint32_t tmem_base = tmem_base_sh;

  if (warp == 0) {
    // ---------------- producer
    if (lane == 0) mbar_expect_tx(&q_full, (uint32_t)(nk * LP_CHUNK_Q));
    __syncwarp();
    if (lane < nk) tma_load_3d(q_s + lane * LP_CHUNK_Q, &map_q, &q_full, (c_lo + lane) * 64, h, row0);
    const int u = lane & 3, slot = lane >> 2;              // unit of 16 keys, place in the stage
    const bool is_v = !shared_row && slot >= prm.k_slots;
    const bool active = is_v ? slot < n_slots : slot < nk;
    const int x = is_v ? (slot - prm.k_slots) * 64 : (c_lo + slot) * 64;
    const uint32_t tile_bytes = (uint32_t)((nk + (shared_row ? 0 : nv)) * LP_CHUNK_K);
    auto unit_row = [&](int it) -> int {
      if (!active || it >= n_it) return 0;
      const bool in_pool = it < n_pool;
      int j;
      if (in_pool) {
        j = min(it * LP_BN + u * LP_UNIT, nb_last - 1) / LP_UNIT * LP_UNIT;
      } else {
        j = min((tile_first + it) * LP_BN + u * LP_UNIT, pos_last) / LP_UNIT * LP_UNIT;
        if (j + LP_UNIT - 1 < key_lo) j = key_lo / LP_UNIT * LP_UNIT;    // (behind the window: its page may be gone)
      }
      const int page = (in_pool ? pool_table : table)[j / prm.page_size];
      if (page < 0 || page >= prm.n_pages) {
        *prm.status = NIB_STATUS_BAD_PAGE;
        return 0;                                          // (page 0: in the pool)
      }
      return ((page * prm.planes + (is_v ? 1 : 0)) * prm.n_kv_head + hk) * prm.page_size + j % prm.page_size;
    };
    bool ok = true;
    int row_next = unit_row(0);
    uint8_t* dst = k_s + slot * LP_CHUNK_K + u * (LP_UNIT * 128);
    for (int it = 0; it < n_it; ++it) {
      const int st = it % stages, round = it / stages;
      const int row = row_next;
      row_next = unit_row(it + 1);    // the next tile's look-up travels while this tile's stage is waited for
      if (round > 0) ok = warp_mbar_wait(&k_empty[st], (round + 1) & 1, abort_flag, lane);
      if (!ok) break;
      if (lane == 0) mbar_expect_tx(&k_full[st], tile_bytes);
      __syncwarp();
      if (active) tma_load_2d(dst + st * stage_bytes, &map_kv, &k_full[st], x, row);
    }
    __syncwarp();
  } else if (warp == 1) {
    // ---------------- MMA issue
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc(LP_BM, LP_BN);
      const uint32_t idesc_o = umma_idesc(LP_BM, nv * 64) | (1u << 16);   // B (= V) is MN-major: keys down the rows
      const uint32_t o_tmem = tmem_base + LP_O_COL;
      const uint32_t qa = smem_u32(q_s);
      auto issue_s = [&](int it) {
        tc_fence_after();
        const uint32_t kb = smem_u32(k_s + (it % stages) * stage_bytes);
        for (int ks = ks_lo; ks < ks_hi; ++ks) {   // 16 values per instruction: 32 bytes along a chunk's row
          const int c = ks / 4 - c_lo, k = ks & 3;
          umma_bf16(tmem_base + (uint32_t)((it % LP_NBUF) * LP_BN), umma_desc(qa + c * LP_CHUNK_Q + k * 32),
                    umma_desc(kb + c * LP_CHUNK_K + k * 32), idesc_s, ks > ks_lo ? 1u : 0u);
        }
        umma_commit(&s_full[it % LP_NBUF]);
      };
      // (V's chunks lie LP_CHUNK_K bytes apart along the values: that is the descriptor's leading byte offset)
      const uint64_t lead = (uint64_t)(LP_CHUNK_K >> 4) << 16;
      auto v_desc = [&](uint32_t addr) { return (umma_desc(addr) & ~(0x3fffull << 16)) | lead; };
      auto issue_pv = [&](int it) {
        tc_fence_after();
        const int st = it % stages, b = it % LP_NBUF;
        const uint32_t vb = smem_u32(k_s + st * stage_bytes + v_off), pa = smem_u32(p_s + b * LP_P_BYTES);
#pragma unroll
        for (int k = 0; k < LP_BN / 16; ++k)   // 16 keys per instruction: P 32 bytes along its row, V 16 rows down
          umma_bf16(o_tmem, umma_desc(pa + k * 32), v_desc(vb + k * 2048), idesc_o, (it > 0 || k > 0) ? 1u : 0u);
        umma_commit(&o_full[b]);
        umma_commit(&k_empty[st]);
      };
      bool ok = mbar_wait(&q_full, 0, abort_flag);
      int s_next = 0, pv_next = 0;
      long long t0 = clock64();
      while (ok && pv_next < n_it) {
        if (pv_next < s_next && lp_test(&p_full[pv_next % LP_NBUF], (pv_next / LP_NBUF) & 1)) {
          issue_pv(pv_next++);
          t0 = clock64();
        } else if (s_next < n_it && s_next < pv_next + LP_NBUF && lp_test(&k_full[s_next % stages], (s_next / stages) & 1)) {
          // (the score buffer is free: P of two tiles ago was made from it, or its P V would not have been issued)
          issue_s(s_next++);
          t0 = clock64();
        } else if (*abort_flag) {
          ok = false;
        } else if (clock64() - t0 > TC_WAIT_CYCLES) {
          *abort_flag = 1;
          ok = false;
        }
      }
    }
    __syncwarp();
  } else {
    // ---------------- softmax: a thread per row; warp w owns tensor-memory lanes 32 * (w % 4) .. +32
    const int quarter = warp & 3;
    const int r = quarter * 32 + lane;
    const uint32_t lane_addr = tmem_base + ((uint32_t)(quarter * 32) << 16);
    const int p = pos_first + r;
    const int lo = (window > 0 && p - window + 1 > 0) ? p - window + 1 : 0;
    const int wp0 = pos_first + quarter * 32, wp1 = wp0 + 31;   // positions of the warp's rows
    const int nb = pooled_blocks_seen(p, window, prm.pool), wnb0 = pooled_blocks_seen(wp0, window, prm.pool);
    constexpr float LOG2E = 1.4426950408889634f;
    const bool capped = prm.softcap > 0.0f;
    const float scale2 = capped ? 1.0f : prm.scale * LOG2E;    // (capped scores are brought to their final form first)
    const float cap2 = prm.softcap * LOG2E, cap_in = capped ? 2.0f * LOG2E * prm.scale / prm.softcap : 0.0f;
    float m = -INFINITY, l = 0.0f;
    bool ok = true;
    for (int it = 0; it < n_it; ++it) {
      const int b = it % LP_NBUF;
      ok = warp_mbar_wait(&s_full[b], (it / LP_NBUF) & 1, abort_flag, lane);
      if (!ok) break;
      tc_fence_after();
      const bool in_pool = it < n_pool;
      const int j0 = in_pool ? it * LP_BN : (tile_first + it) * LP_BN;
      // a row sees the keys first .. last of the tile's kind; only tiles at an edge need the mask
      const int first = in_pool ? 0 : lo, last = in_pool ? nb - 1 : p;
      const bool edge = in_pool ? j0 + LP_BN > wnb0 : j0 + LP_BN - 1 > wp0 || (window > 0 && j0 < wp1 - window + 1);
      float v[LP_BN];
#pragma unroll
      for (int c = 0; c < LP_BN / 32; ++c) lp_tmem_ld32(lane_addr + (uint32_t)(b * LP_BN + c * 32), v + c * 32);
      if (capped) {
        // c tanh(x / c) by tanh(y) = 1 - 2 / (1 + e^2y) with the hardware's 2^x and division: relative error about 1e-6
#pragma unroll
        for (int i = 0; i < LP_BN; ++i) v[i] = cap2 - __fdividef(2.0f * cap2, 1.0f + lp_pow2(v[i] * cap_in));
      }
      if (edge) {
#pragma unroll
        for (int i = 0; i < LP_BN; ++i)
          if (!(j0 + i <= last && j0 + i >= first)) v[i] = -INFINITY;
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};   // four chains, not one of 64 links
#pragma unroll
      for (int i = 0; i < LP_BN; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], v[i]);
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * scale2;   // (scale2 > 0)
      const bool raise = it == 0 || __any_sync(0xffffffffu, mx > m + LP_RAISE || (m == -INFINITY && mx > m));
      if (raise) {
        const float m_new = fmaxf(m, mx);
        if (it > 0) {
          const float corr = (m_new == -INFINITY) ? 1.0f : lp_pow2(m - m_new);
          l *= corr;
          // O holds the tiles up to it - 1 once their MMAs are done
          ok = warp_mbar_wait(&o_full[(it - 1) % LP_NBUF], ((it - 1) / LP_NBUF) & 1, abort_flag, lane);
          if (!ok) break;
          tc_fence_after();
#pragma unroll 1
          for (int c = 0; c < nv * 4; ++c) {
            float t[16];
            tmem_ld16(lane_addr + LP_O_COL + (uint32_t)(c * 16), t);
#pragma unroll
            for (int i = 0; i < 16; ++i) t[i] *= corr;
            lp_tmem_st16(lane_addr + LP_O_COL + (uint32_t)(c * 16), t);
          }
          asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        }
        m = m_new;
      }
      const float ms = (m == -INFINITY) ? 0.0f : m;     // (a row with no key yet: 2^(-inf - -inf) is avoided)
      // P of tile it - 2 (the last user of this buffer) has been read by its MMA
      if (it >= LP_NBUF) {
        ok = warp_mbar_wait(&o_full[b], ((it - LP_NBUF) / LP_NBUF) & 1, abort_flag, lane);
        if (!ok) break;
      }
      float sum4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
      uint8_t* blk = p_s + b * LP_P_BYTES + r * 128;
#pragma unroll
      for (int g = 0; g < LP_BN / 8; ++g) {
        float e8[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          e8[i] = lp_pow2(fmaf(v[8 * g + i], scale2, -ms));   // 0 for a masked key
          sum4[i & 3] += e8[i];
        }
        *reinterpret_cast<uint4*>(blk + ((g ^ (r & 7)) * 16)) =
            make_uint4(pack_bf16(e8[0], e8[1]), pack_bf16(e8[2], e8[3]), pack_bf16(e8[4], e8[5]), pack_bf16(e8[6], e8[7]));
      }
      l += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");   // generic writes -> visible to the MMAs
      tc_fence_before();
      asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(&p_full[b])) : "memory");
    }
    // the last MMA into O
    if (ok) ok = warp_mbar_wait(&o_full[(n_it - 1) % LP_NBUF], ((n_it - 1) / LP_NBUF) & 1, abort_flag, lane);
    if (ok) {
      tc_fence_after();
      if (prm.sinks != nullptr) l += lp_pow2(prm.sinks[h] * LOG2E - m);
      float inv = l > 0.0f ? 1.0f / l : 0.0f;
      if (prm.gate != nullptr && prm.gate_dim == 0 && r < n_rows) inv *= 1.0f / (1.0f + __expf(-prm.gate[(size_t)(row0 + r) * prm.ldg + h]));
      const size_t at = (size_t)(row0 + r) * prm.ldo + (size_t)h * prm.out_head;
      bf16* dst = reinterpret_cast<bf16*>(prm.out) + at;
      float* dst32 = reinterpret_cast<float*>(prm.out) + at;
#pragma unroll 1
      for (int c = 0; c < nv * 4; ++c) {
        float t[16];
        tmem_ld16(lane_addr + LP_O_COL + (uint32_t)(c * 16), t);
        if (r < n_rows) {
          if (prm.gate_dim > 0) {
            const float* gr = prm.gate + (size_t)(row0 + r) * prm.ldg + h * prm.gate_dim + c * 16;
            const int left = prm.gate_dim - c * 16;
            if (left >= 16 && ((uintptr_t)gr & 15) == 0) {
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                const float4 g4 = reinterpret_cast<const float4*>(gr)[i];
                t[4 * i] *= lp_sigmoid(g4.x); t[4 * i + 1] *= lp_sigmoid(g4.y);
                t[4 * i + 2] *= lp_sigmoid(g4.z); t[4 * i + 3] *= lp_sigmoid(g4.w);
              }
            } else {
#pragma unroll
              for (int i = 0; i < 16; ++i)
                if (i < left) t[i] *= lp_sigmoid(gr[i]);
            }
          }
#pragma unroll
          for (int g = 0; g < 2; ++g) {
            const int d = c * 16 + 8 * g;
            if (d >= prm.v_cols) continue;          // (v_cols is a multiple of 8)
            if (prm.out32) {
              *reinterpret_cast<float4*>(dst32 + d) = make_float4(t[8 * g] * inv, t[8 * g + 1] * inv, t[8 * g + 2] * inv, t[8 * g + 3] * inv);
              *reinterpret_cast<float4*>(dst32 + d + 4) =
                  make_float4(t[8 * g + 4] * inv, t[8 * g + 5] * inv, t[8 * g + 6] * inv, t[8 * g + 7] * inv);
            } else {
              *reinterpret_cast<uint4*>(dst + d) =
                  make_uint4(pack_bf16(t[8 * g] * inv, t[8 * g + 1] * inv), pack_bf16(t[8 * g + 2] * inv, t[8 * g + 3] * inv),
                             pack_bf16(t[8 * g + 4] * inv, t[8 * g + 5] * inv), pack_bf16(t[8 * g + 6] * inv, t[8 * g + 7] * inv));
            }
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (threadIdx.x == 0 && abort_sh) *prm.status = NIB_STATUS_WAIT_TIMEOUT;
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, LP_TMEM_COLS);
  }
}

// Q as [T rows][heads][row_dim values], moved in boxes of 128 rows x 1 head x 64 values; what lies beyond reads as zeros.
static bool make_q_map(CUtensorMap* map, const void* base, int ldq, int T, int n_head, int row_dim) {
  EncodeTiledFn fn = encode_fn();
  if (!fn) return false;
  cuuint64_t dims[3] = {(cuuint64_t)row_dim, (cuuint64_t)n_head, (cuuint64_t)T};
  cuuint64_t strides[2] = {(cuuint64_t)row_dim * 2, (cuuint64_t)ldq * 2};
  cuuint32_t box[3] = {64, 1, LP_BM};
  cuuint32_t estr[3] = {1, 1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// chunks of 64 values that the keys of any map of a row touch (whole steps of 16 values)
static int lp_key_chunks(int maps, int map_dim) {
  int most = 0;
  for (int m = 0; m < maps; ++m) {
    const int lo = m * map_dim / 16, hi = ((m + 1) * map_dim + 15) / 16;
    const int n = (hi + 3) / 4 - lo / 4;
    if (n > most) most = n;
  }
  return most;
}
static size_t lp_smem(int k_slots, int v_slots, int stages) {
  return (size_t)k_slots * LP_CHUNK_Q + (size_t)stages * (k_slots + v_slots) * LP_CHUNK_K + (size_t)LP_NBUF * LP_P_BYTES + 1024;
}
constexpr size_t LP_MAX_SMEM = 225 * 1024;

}  // namespace nib

using namespace nib;

// 1 if the kernel takes these sizes: rows of a multiple of 8 values, v_cols a multiple of 8 up to 256, pages of a multiple of
// 16 positions, two stages within shared memory.
extern "C" int nib_attention_wide_tc_supported(int row_dim, int planes, int maps, int map_dim, int v_cols, int page_size) {
  if (row_dim <= 0 || row_dim % 8 || (planes != 1 && planes != 2) || maps <= 0 || map_dim <= 0 || maps * map_dim > row_dim) return 0;
  if (v_cols <= 0 || v_cols % 8 || v_cols > row_dim || v_cols > 64 * LP_MAX_V_CHUNKS) return 0;
  if (page_size < LP_UNIT || page_size % LP_UNIT) return 0;
  const int nv = (v_cols + 63) / 64, nk = lp_key_chunks(maps, map_dim), vs = planes == 1 ? 0 : nv;
  if (planes == 1 && (maps != 1 || map_dim != row_dim)) return 0;
  return nk + vs <= LP_MAX_SLOTS && lp_smem(nk, vs, 2) <= LP_MAX_SMEM;
}

// tiles: n_tiles pairs (entry, first row within the entry), 128 rows each (the last of an entry may be shorter).  q [T rows,
// ldq], heads of row_dim values one after the other; cache: one layer [n_pages, planes, n_kv_head, page_size, row_dim]; out:
// head h's v_cols values at column h * out_head of its rows (ldo elements apart), bfloat16 or with out32 32-bit floats.
extern "C" int nib_attention_wide_tc(const void* q, int ldq, int T, const void* cache, int planes, void* out, int ldo,
                                     int out_head, int out32, const int* block_table, int max_blocks, const int* tiles,
                                     int n_tiles, const int* entry_start, const int* entry_pos0, int n_head, int n_kv_head,
                                     int row_dim, int maps, int map_dim, int v_cols, int page_size, int n_pages, float scale,
                                     int window, float softcap, const float* gate, int ldg, int gate_dim, const float* sinks,
                                     int pool, const int* pool_table, int* status, cudaStream_t stream) {
  if (n_tiles <= 0) return 0;
  if (!nib_attention_wide_tc_supported(row_dim, planes, maps, map_dim, v_cols, page_size)) return NIB_ERR_UNSUPPORTED_SIZE;
  if (n_head <= 0 || n_kv_head <= 0 || n_head % n_kv_head || T <= 0 || !(scale > 0.0f) || softcap < 0.0f)
    return NIB_ERR_BAD_ARGUMENT;
  if (pool < 0 || gate_dim < 0 || (pool > 0 && (window <= 0 || pool_table == nullptr)) || (gate_dim > 0 && gate == nullptr))
    return NIB_ERR_BAD_ARGUMENT;
  const int align = out32 ? 3 : 7;
  if (((uintptr_t)q & 15) || ((uintptr_t)cache & 15) || ((uintptr_t)out & 15) || (ldo & align) || (out_head & align) || (ldq & 7))
    return NIB_ERR_UNSUPPORTED_SIZE;
  const long long kv_rows = (long long)n_pages * planes * n_kv_head * page_size;
  if (n_tiles > 65535 || kv_rows > 0x7fffffffll) return NIB_ERR_UNSUPPORTED_SIZE;
  CUtensorMap map_q, map_kv;
  if (!make_q_map(&map_q, q, ldq, T, n_head, row_dim)) return NIB_ERR_DRIVER;
  if (!make_map(&map_kv, cache, false, (int)kv_rows, row_dim, row_dim, LP_UNIT, 64, true)) return NIB_ERR_DRIVER;
  LpParams prm;
  prm.block_table = block_table; prm.max_blocks = max_blocks; prm.tiles = tiles;
  prm.entry_start = entry_start; prm.entry_pos0 = entry_pos0; prm.page_size = page_size; prm.n_pages = n_pages;
  prm.n_head = n_head; prm.n_kv_head = n_kv_head; prm.planes = planes;
  prm.row_dim = row_dim; prm.maps = maps; prm.map_dim = map_dim;
  prm.v_cols = v_cols; prm.v_chunks = (v_cols + 63) / 64; prm.k_slots = lp_key_chunks(maps, map_dim);
  const int vs = planes == 1 ? 0 : prm.v_chunks;
  prm.stages = 2;
  while (prm.stages < LP_MAX_STAGES && lp_smem(prm.k_slots, vs, prm.stages + 1) <= LP_MAX_SMEM) ++prm.stages;
  prm.scale = scale; prm.softcap = softcap; prm.window = window; prm.gate = gate; prm.ldg = ldg;
  prm.gate_dim = gate_dim; prm.sinks = sinks; prm.pool = pool; prm.pool_table = pool > 0 ? pool_table : block_table;
  prm.out = out; prm.ldo = ldo; prm.out_head = out_head; prm.out32 = out32; prm.status = status;
  static bool attr_set = false;
  if (!attr_set) {
    const cudaError_t err = cudaFuncSetAttribute(attention_wide_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LP_MAX_SMEM);
    if (err != cudaSuccess) return (int)err;
    attr_set = true;
  }
  launch_pdl(attention_wide_tc_kernel, dim3(n_head, n_tiles), dim3(LP_THREADS), lp_smem(prm.k_slots, vs, prm.stages), stream,
             map_q, map_kv, prm);
  NIB_LAUNCH_CHECK();
}
