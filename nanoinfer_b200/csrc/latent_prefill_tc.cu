// Attention through a low-rank latent for prompt portions, on the fifth-generation tensor cores (bfloat16).
//
// A head's query has been carried into the latent space (latent_attention.cu says how), so that every head attends over
// the same cached rows [c | k_rot] of D values, and the weighted sum is over their first kv_rank values: one tile of the
// cache is both the keys and the values.  One block takes 128 consecutive query rows of one request and one head and
// walks the keys in tiles of 64:
//   warp 0      the producer: Q once; then a tile of the cache at a time, 16 rows x 64 values a TMA load (a lane each, with
//               its own look-up in the block table), into a ring of stages of 128-byte-swizzled shared memory, a stage
//               being D / 64 chunks of [64 keys][64 values];
//   warp 1      the MMAs: S = Q K^T (128 x 64 x D) into one of two score buffers in tensor memory; O += P V (128 x kv_rank x
//               64) with P from shared memory and V the same stage read as an MN-major operand (keys down the rows, chunks of
//               64 values side by side), accumulated in tensor memory over all tiles.  A stage is free when its P V is done;
//   warps 2..5  the softmax, a thread a row: scores times log2(e), running maximum raised only when a tile exceeds it by
//               more than 2^8 (O is then scaled in tensor memory), P as bfloat16, the sum in 32-bit; at the end the
//               division, the head's gate, and the store.
// Keys outside [lowest visible, last row] are masked; their rows are read from the nearest unit of the request that is
// there.  What a box reaches beyond D, or beyond the step's rows, reads as zeros.
//
// Every wait on a barrier is bounded: a wait that runs out sets the block's abort flag and the device status word, every
// role leaves its loop, tensor memory is freed, and the kernel returns.
#include "api.h"
#include "common.cuh"
#include "tcgen05.cuh"

namespace nib {

constexpr int LP_BM = 128, LP_BN = 64, LP_UNIT = 16, LP_THREADS = 192, LP_NBUF = 2, LP_MAX_STAGES = 4;
constexpr int LP_MAX_CHUNKS = 5, LP_MAX_V_CHUNKS = 4;        // D <= 320, kv_rank <= 256
constexpr int LP_CHUNK_Q = LP_BM * 128, LP_CHUNK_K = LP_BN * 128, LP_P_BYTES = LP_BM * 128;
constexpr uint32_t LP_O_COL = LP_NBUF * LP_BN, LP_TMEM_COLS = 512;
constexpr float LP_RAISE = 8.0f;

struct LpParams {
  const int* block_table;
  int max_blocks;
  const int* tiles;            // pairs (entry, first row within the entry), 128 rows each
  const int* entry_start;
  const int* entry_pos0;
  int page_size, n_pages;
  int kv_rank, n_chunks, v_chunks, stages;
  float scale;
  int window;
  const float* gate;
  int ldg;
  bf16* out;
  int ldo;
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

__global__ void __launch_bounds__(LP_THREADS, 1)
latent_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv,
                         const LpParams prm) {
  extern __shared__ uint8_t lp_smem_raw[];
  // tiles must start on a 1024-byte boundary for the 128-byte swizzle
  uint8_t* smem = reinterpret_cast<uint8_t*>(((uintptr_t)lp_smem_raw + 1023) & ~(uintptr_t)1023);
  const int nk = prm.n_chunks, nv = prm.v_chunks, stages = prm.stages;
  const int stage_bytes = nk * LP_CHUNK_K;
  uint8_t* q_s = smem;                                  // [chunks][128 rows][64]
  uint8_t* k_s = q_s + nk * LP_CHUNK_Q;                 // [stages][chunks][64 keys][64]
  uint8_t* p_s = k_s + stages * stage_bytes;            // [2][128 rows][64 keys]
  __shared__ __align__(8) uint64_t q_full, k_full[LP_MAX_STAGES], k_empty[LP_MAX_STAGES], s_full[LP_NBUF], p_full[LP_NBUF],
      o_full[LP_NBUF];
  __shared__ uint32_t tmem_base_sh;
  __shared__ int abort_sh;
  volatile int* abort_flag = &abort_sh;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // (heads are the fast index of the grid: blocks start in the order of the tile list, longest first)
  const int e = prm.tiles[2 * blockIdx.y], q_off = prm.tiles[2 * blockIdx.y + 1];
  const int h = blockIdx.x;
  const int row0 = prm.entry_start[e] + q_off;                    // first row of the tile in the step
  const int n_rows = min(LP_BM, prm.entry_start[e + 1] - row0);
  const int pos_first = prm.entry_pos0[e] + q_off;                // position of the tile's first row
  const int pos_last = pos_first + n_rows - 1;
  const int* table = prm.block_table + (size_t)e * prm.max_blocks;
  const int window = prm.window;
  const int key_lo = (window > 0 && pos_first - window + 1 > 0) ? pos_first - window + 1 : 0;
  const int tile_first = key_lo / LP_BN, n_it = pos_last / LP_BN - tile_first + 1;

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
    if (lane < nk) tma_load_3d(q_s + lane * LP_CHUNK_Q, &map_q, &q_full, lane * 64, h, row0);
    const int u = lane & 3, chunk = lane >> 2;             // unit of 16 keys, chunk of 64 values
    const bool active = chunk < nk;
    auto unit_row = [&](int it) -> int {
      if (!active || it >= n_it) return 0;
      int j = min((tile_first + it) * LP_BN + u * LP_UNIT, pos_last) / LP_UNIT * LP_UNIT;
      if (j + LP_UNIT - 1 < key_lo) j = key_lo / LP_UNIT * LP_UNIT;      // (behind the window: its page may be gone)
      const int page = table[j / prm.page_size];
      if (page < 0 || page >= prm.n_pages) {
        *prm.status = NIB_STATUS_BAD_PAGE;
        return 0;                                          // (page 0: in the pool)
      }
      return page * prm.page_size + j % prm.page_size;
    };
    bool ok = true;
    int row_next = unit_row(0);
    uint8_t* dst = k_s + chunk * LP_CHUNK_K + u * (LP_UNIT * 128);
    for (int it = 0; it < n_it; ++it) {
      const int st = it % stages, round = it / stages;
      const int row = row_next;
      row_next = unit_row(it + 1);    // the next tile's look-up travels while this tile's stage is waited for
      if (round > 0) ok = warp_mbar_wait(&k_empty[st], (round + 1) & 1, abort_flag, lane);
      if (!ok) break;
      if (lane == 0) mbar_expect_tx(&k_full[st], (uint32_t)stage_bytes);
      __syncwarp();
      if (active) tma_load_2d(dst + st * stage_bytes, &map_kv, &k_full[st], chunk * 64, row);
    }
    __syncwarp();
  } else if (warp == 1) {
    // ---------------- MMA issue
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc(LP_BM, LP_BN);
      const uint32_t idesc_o = umma_idesc(LP_BM, nv * 64) | (1u << 16);   // B (= V) is MN-major: keys down the rows
      const uint32_t o_tmem = tmem_base + LP_O_COL;
      const uint32_t qa = smem_u32(q_s);
      auto issue_s = [&](int it) -> bool {
        const int st = it % stages;
        if (!mbar_wait(&k_full[st], (it / stages) & 1, abort_flag)) return false;
        tc_fence_after();
        const uint32_t kb = smem_u32(k_s + st * stage_bytes);
        for (int c = 0; c < nk; ++c)
#pragma unroll
          for (int k = 0; k < 4; ++k)   // 16 of a chunk's 64 values per instruction: 32 bytes along the row
            umma_bf16(tmem_base + (uint32_t)((it % LP_NBUF) * LP_BN), umma_desc(qa + c * LP_CHUNK_Q + k * 32),
                      umma_desc(kb + c * LP_CHUNK_K + k * 32), idesc_s, (c > 0 || k > 0) ? 1u : 0u);
        umma_commit(&s_full[it % LP_NBUF]);
        return true;
      };
      // (V's chunks lie LP_CHUNK_K bytes apart along the values: that is the descriptor's leading byte offset)
      const uint64_t lead = (uint64_t)(LP_CHUNK_K >> 4) << 16;
      auto v_desc = [&](uint32_t addr) { return (umma_desc(addr) & ~(0x3fffull << 16)) | lead; };
      bool ok = mbar_wait(&q_full, 0, abort_flag);
      for (int a = 0; ok && a < LP_NBUF && a < n_it; ++a) ok = issue_s(a);
      for (int it = 0; ok && it < n_it; ++it) {
        const int st = it % stages, b = it % LP_NBUF;
        if (!mbar_wait(&p_full[b], (it / LP_NBUF) & 1, abort_flag)) break;
        tc_fence_after();
        const uint32_t vb = smem_u32(k_s + st * stage_bytes), pa = smem_u32(p_s + b * LP_P_BYTES);
#pragma unroll
        for (int k = 0; k < LP_BN / 16; ++k)   // 16 keys per instruction: P 32 bytes along its row, V 16 rows down
          umma_bf16(o_tmem, umma_desc(pa + k * 32), v_desc(vb + k * 2048), idesc_o, (it > 0 || k > 0) ? 1u : 0u);
        umma_commit(&o_full[b]);
        umma_commit(&k_empty[st]);
        if (it + LP_NBUF < n_it) ok = issue_s(it + LP_NBUF);
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
    const float scale2 = prm.scale * 1.4426950408889634f;
    float m = -INFINITY, l = 0.0f;
    bool ok = true;
    for (int it = 0; it < n_it; ++it) {
      const int b = it % LP_NBUF;
      ok = warp_mbar_wait(&s_full[b], (it / LP_NBUF) & 1, abort_flag, lane);
      if (!ok) break;
      tc_fence_after();
      const int j0 = (tile_first + it) * LP_BN;
      const bool edge = j0 + LP_BN - 1 > wp0 || (window > 0 && j0 < wp1 - window + 1);   // only these tiles need the mask
      float v[LP_BN];
#pragma unroll
      for (int c = 0; c < LP_BN / 32; ++c) lp_tmem_ld32(lane_addr + (uint32_t)(b * LP_BN + c * 32), v + c * 32);
      if (edge) {
#pragma unroll
        for (int i = 0; i < LP_BN; ++i)
          if (!(j0 + i <= p && j0 + i >= lo)) v[i] = -INFINITY;
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
      float inv = l > 0.0f ? 1.0f / l : 0.0f;
      if (prm.gate != nullptr && r < n_rows) inv *= 1.0f / (1.0f + __expf(-prm.gate[(size_t)(row0 + r) * prm.ldg + h]));
      bf16* dst = prm.out + (size_t)(row0 + r) * prm.ldo + (size_t)h * prm.kv_rank;
#pragma unroll 1
      for (int c = 0; c < nv * 4; ++c) {
        float t[16];
        tmem_ld16(lane_addr + LP_O_COL + (uint32_t)(c * 16), t);
        if (r < n_rows) {
#pragma unroll
          for (int g = 0; g < 2; ++g)
            if (c * 16 + 8 * g < prm.kv_rank)       // (kv_rank is a multiple of 8)
              *reinterpret_cast<uint4*>(dst + c * 16 + 8 * g) =
                  make_uint4(pack_bf16(t[8 * g] * inv, t[8 * g + 1] * inv), pack_bf16(t[8 * g + 2] * inv, t[8 * g + 3] * inv),
                             pack_bf16(t[8 * g + 4] * inv, t[8 * g + 5] * inv), pack_bf16(t[8 * g + 6] * inv, t[8 * g + 7] * inv));
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

// Q as [T rows][heads][D values], moved in boxes of 128 rows x 1 head x 64 values; what lies beyond D or T reads as zeros.
static bool make_q_map(CUtensorMap* map, const void* base, int T, int n_head, int D) {
  EncodeTiledFn fn = encode_fn();
  if (!fn) return false;
  cuuint64_t dims[3] = {(cuuint64_t)D, (cuuint64_t)n_head, (cuuint64_t)T};
  cuuint64_t strides[2] = {(cuuint64_t)D * 2, (cuuint64_t)n_head * D * 2};
  cuuint32_t box[3] = {64, 1, LP_BM};
  cuuint32_t estr[3] = {1, 1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

static size_t lp_smem(int n_chunks, int stages) {
  return (size_t)n_chunks * LP_CHUNK_Q + (size_t)stages * n_chunks * LP_CHUNK_K + (size_t)LP_NBUF * LP_P_BYTES + 1024;
}

}  // namespace nib

using namespace nib;

// 1 if the kernel takes these sizes: D a multiple of 8 up to 320, kv_rank a multiple of 8 up to 256, pages of a multiple
// of 16 positions.
extern "C" int nib_latent_prefill_tc_supported(int kv_rank, int D, int page_size) {
  return D % 8 == 0 && D <= 64 * LP_MAX_CHUNKS && kv_rank % 8 == 0 && kv_rank > 0 && kv_rank <= 64 * LP_MAX_V_CHUNKS &&
         kv_rank <= D && page_size >= LP_UNIT && page_size % LP_UNIT == 0;
}

// tiles: n_tiles pairs (entry, first row within the entry), 128 rows each (the last of an entry may be shorter).  q [T,
// n_head, D] contiguous bfloat16; cache: one layer [n_pages, page_size, D]; out rows of n_head * kv_rank values, 16-byte
// aligned.
extern "C" int nib_latent_prefill_tc(const void* q, int T, const void* cache, void* out, int ldo, const int* block_table,
                                     int max_blocks, const int* tiles, int n_tiles, const int* entry_start,
                                     const int* entry_pos0, int n_head, int kv_rank, int D, int page_size, int n_pages,
                                     float scale, int window, const float* gate, int ldg, int* status,
                                     cudaStream_t stream) {
  if (n_tiles <= 0) return 0;
  if (!nib_latent_prefill_tc_supported(kv_rank, D, page_size)) return NIB_ERR_UNSUPPORTED_SIZE;
  if (n_head <= 0 || T <= 0 || !(scale > 0.0f)) return NIB_ERR_BAD_ARGUMENT;
  if (((uintptr_t)q & 15) || ((uintptr_t)cache & 15) || ((uintptr_t)out & 15) || (ldo & 7)) return NIB_ERR_UNSUPPORTED_SIZE;
  const long long kv_rows = (long long)n_pages * page_size;
  if (n_tiles > 65535 || kv_rows > 0x7fffffffll) return NIB_ERR_UNSUPPORTED_SIZE;
  CUtensorMap map_q, map_kv;
  if (!make_q_map(&map_q, q, T, n_head, D)) return NIB_ERR_DRIVER;
  if (!make_map(&map_kv, cache, false, (int)kv_rows, D, D, LP_UNIT, 64, true)) return NIB_ERR_DRIVER;
  LpParams prm;
  prm.block_table = block_table; prm.max_blocks = max_blocks; prm.tiles = tiles;
  prm.entry_start = entry_start; prm.entry_pos0 = entry_pos0; prm.page_size = page_size; prm.n_pages = n_pages;
  prm.kv_rank = kv_rank; prm.n_chunks = (D + 63) / 64; prm.v_chunks = (kv_rank + 63) / 64;
  prm.stages = 2;
  while (prm.stages < LP_MAX_STAGES && lp_smem(prm.n_chunks, prm.stages + 1) <= 220 * 1024) ++prm.stages;
  prm.scale = scale; prm.window = window; prm.gate = gate; prm.ldg = ldg; prm.out = (bf16*)out; prm.ldo = ldo;
  prm.status = status;
  const size_t smem = lp_smem(prm.n_chunks, prm.stages);
  static bool attr_set = false;
  if (!attr_set) {
    const cudaError_t err = cudaFuncSetAttribute(latent_prefill_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 225 * 1024);
    if (err != cudaSuccess) return (int)err;
    attr_set = true;
  }
  launch_pdl(latent_prefill_tc_kernel, dim3(n_head, n_tiles), dim3(LP_THREADS), smem, stream, map_q, map_kv, prm);
  NIB_LAUNCH_CHECK();
}
