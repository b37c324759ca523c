// Attention through a low-rank latent for single decoded tokens in bfloat16, on warp-level MMAs.
//
// All heads of a row attend over the same cached rows [c | k_rot] of D values (latent_attention.cu), so sixteen heads are
// the rows of one MMA tile: S = Q K^T and O += P V read a tile of 64 cached rows once from shared memory for sixteen heads.
// One block takes a row, a group of sixteen heads and a piece of the row's keys.  Per tile: four warps make the scores of
// sixteen keys each (m16n8k16 over D), the row maxima and sums meet in shared memory, P lies there as bfloat16, and every
// warp adds P V for its share of the kv_rank values.  Tiles come through two buffers by cp.async, the first of them ahead
// of griddepcontrol.wait where it does not hold the row's own key.  The pieces of a row are the blocks of one cluster: each
// leaves its (maximum, sum, unscaled result) in its own shared memory, and every block merges its share of the values out
// of all of them through distributed shared memory, in the order of the pieces.  Scores, softmax and sums are 32-bit.
#include "api.h"
#include "common.cuh"

namespace nib {

constexpr int LM_HEADS = 16, LM_BN = 64, LM_WARPS = 4, LM_MAX_SPLITS = 16;

__device__ __forceinline__ void lm_ldmatrix_x4(uint32_t* r, const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void lm_ldmatrix_x4_trans(uint32_t* r, const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void lm_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float lm_pow2(float x) {   // the hardware's 2^x (relative error about 2^-22; 2^-inf = 0)
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// NP: groups of sixteen values of the result that a warp owns (kv_rank <= 64 NP)
template <int NP>
__global__ void __launch_bounds__(LM_WARPS * 32)
latent_decode_mma_kernel(const bf16* q, const bf16* cache, bf16* out, int ldo, const int* __restrict__ block_table,
                         int max_blocks, const int* __restrict__ rows, const int* __restrict__ row_entry,
                         const int* __restrict__ positions, int n_head, int kv_rank, int D, int page_size, int n_pages,
                         float scale, int window, const float* gate, int ldg, int* status, int n_splits) {
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t lm_smem[];
  const int Dk = (D + 15) & ~15, LD = Dk + 8, CH = Dk / 8;         // a row in 16-byte pieces, padded against bank conflicts
  bf16* qs = reinterpret_cast<bf16*>(lm_smem);                      // [16][LD]
  bf16* ks = qs + LM_HEADS * LD;                                    // [2][64][LD]
  bf16* ps = ks + 2 * LM_BN * LD;                                   // [16][72]
  float* red = reinterpret_cast<float*>(ps + LM_HEADS * 72);        // [2][4 warps][16]
  float* stats = red + 2 * LM_WARPS * LM_HEADS;                     // [16][2]: this piece's maximum and sum
  float* all = stats + 2 * LM_HEADS;                                // [splits][16][2]
  float* xo = reinterpret_cast<float*>(ks);                         // [16][kv_rank], behind the last tile
  const int split = blockIdx.x, h0 = blockIdx.y * LM_HEADS;
  const int t = rows ? rows[blockIdx.z] : blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int entry = row_entry[t], pos = positions[t];
  // (a row of no request takes part in the cluster's barriers with an empty piece)
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;
  const int per = ((pos - lo + n_splits) / n_splits + 15) / 16 * 16;
  const int k_begin = lo + split * per, k_end = entry < 0 ? 0 : min(pos + 1, k_begin + per);
  const int n_it = k_end > k_begin ? (k_end - k_begin + LM_BN - 1) / LM_BN : 0;
  const int* table = block_table + (size_t)max(entry, 0) * max_blocks;

  const int step_r = (LM_WARPS * 32) / CH, step_p = (LM_WARPS * 32) % CH;
  auto load_tile = [&](int it, int buf) {
    const int j0 = k_begin + it * LM_BN;
    int r = tid / CH, piece = tid % CH, last_r = -1;
    const bf16* row = cache;
    bool there = false;
    while (r < LM_BN) {
      const int j = j0 + r;
      if (r != last_r) {
        there = j < k_end;
        if (there) {
          const int page = table[j / page_size];
          if (page < 0 || page >= n_pages) {
            *status = NIB_STATUS_BAD_PAGE;
            there = false;
          } else {
            row = cache + ((size_t)page * page_size + j % page_size) * (size_t)D;
          }
        }
        last_r = r;
      }
      const bool valid = there && piece * 8 < D;                    // (D is a multiple of 8)
      cp_async16(ks + (buf * LM_BN + r) * LD + piece * 8, valid ? row + piece * 8 : cache, valid);
      r += step_r;
      piece += step_p;
      if (piece >= CH) {
        piece -= CH;
        ++r;
      }
    }
  };
  const bool early = n_it > 0 && min(k_end, k_begin + LM_BN) <= pos;   // the first tile does not hold the row's own key
  if (early) load_tile(0, 0);
  pdl_wait();
  if (n_it > 0) {
    for (int c = tid; c < LM_HEADS * CH; c += LM_WARPS * 32) {
      const int r = c / CH, piece = c % CH;
      const bool valid = h0 + r < n_head && piece * 8 < D;
      const bf16* src = q + ((size_t)t * n_head + (valid ? h0 + r : 0)) * (size_t)D + (valid ? piece * 8 : 0);
      cp_async16(qs + r * LD + piece * 8, src, valid);
    }
    if (!early) load_tile(0, 0);
  }
  cp_async_commit();

  float o[2 * NP][4];
#pragma unroll
  for (int i = 0; i < 2 * NP; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;     // of heads lane / 4 and lane / 4 + 8
  const int r0 = lane >> 2, r1 = r0 + 8, n_pairs = (kv_rank + 15) / 16;
  const float scale2 = scale * 1.4426950408889634f;
  for (int it = 0; it < n_it; ++it) {
    const int buf = it & 1;
    if (it + 1 < n_it) load_tile(it + 1, buf ^ 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    // ---- the scores of this warp's sixteen keys
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    const bf16* kt = ks + (buf * LM_BN + warp * 16) * LD;
    for (int kk = 0; kk < Dk / 16; ++kk) {
      uint32_t a[4], b[4];
      lm_ldmatrix_x4(a, qs + ((lane & 7) + 8 * ((lane >> 3) & 1)) * LD + kk * 16 + 8 * (lane >> 4));
      lm_ldmatrix_x4(b, kt + ((lane & 7) + 8 * (lane >> 4)) * LD + kk * 16 + 8 * ((lane >> 3) & 1));
      lm_mma(s[0], a, b[0], b[1]);
      lm_mma(s[1], a, b[2], b[3]);
    }
    const int j_base = k_begin + it * LM_BN + warp * 16 + (lane & 3) * 2;
    float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const bool live = j_base + i * 8 + c < k_end;
        s[i][c] = live ? s[i][c] * scale2 : -INFINITY;
        s[i][2 + c] = live ? s[i][2 + c] * scale2 : -INFINITY;
        mx0 = fmaxf(mx0, s[i][c]);
        mx1 = fmaxf(mx1, s[i][2 + c]);
      }
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    if ((lane & 3) == 0) {
      red[warp * LM_HEADS + r0] = mx0;
      red[warp * LM_HEADS + r1] = mx1;
    }
    __syncthreads();
    float n0 = m0, n1 = m1;
#pragma unroll
    for (int w = 0; w < LM_WARPS; ++w) {
      n0 = fmaxf(n0, red[w * LM_HEADS + r0]);
      n1 = fmaxf(n1, red[w * LM_HEADS + r1]);
    }
    // (every tile holds at least one live key: n0 and n1 are finite)
    float sum0 = 0.0f, sum1 = 0.0f;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        s[i][c] = lm_pow2(s[i][c] - n0);
        s[i][2 + c] = lm_pow2(s[i][2 + c] - n1);
        sum0 += s[i][c];
        sum1 += s[i][2 + c];
      }
      const int col = warp * 16 + i * 8 + (lane & 3) * 2;
      *reinterpret_cast<__nv_bfloat162*>(ps + r0 * 72 + col) = __floats2bfloat162_rn(s[i][0], s[i][1]);
      *reinterpret_cast<__nv_bfloat162*>(ps + r1 * 72 + col) = __floats2bfloat162_rn(s[i][2], s[i][3]);
    }
    sum0 += __shfl_xor_sync(0xffffffffu, sum0, 1);
    sum0 += __shfl_xor_sync(0xffffffffu, sum0, 2);
    sum1 += __shfl_xor_sync(0xffffffffu, sum1, 1);
    sum1 += __shfl_xor_sync(0xffffffffu, sum1, 2);
    float* sums = red + LM_WARPS * LM_HEADS;
    if ((lane & 3) == 0) {
      sums[warp * LM_HEADS + r0] = sum0;
      sums[warp * LM_HEADS + r1] = sum1;
    }
    __syncthreads();
    const float c0 = lm_pow2(m0 - n0), c1 = lm_pow2(m1 - n1);      // (2^-inf = 0 at the first tile)
    l0 *= c0;
    l1 *= c1;
#pragma unroll
    for (int w = 0; w < LM_WARPS; ++w) {
      l0 += sums[w * LM_HEADS + r0];
      l1 += sums[w * LM_HEADS + r1];
    }
    m0 = n0;
    m1 = n1;
    // ---- O += P V for this warp's values: groups warp, warp + 4, ... of sixteen
    uint32_t pa[4][4];
#pragma unroll
    for (int kk = 0; kk < 4; ++kk)
      lm_ldmatrix_x4(pa[kk], ps + ((lane & 7) + 8 * ((lane >> 3) & 1)) * 72 + kk * 16 + 8 * (lane >> 4));
    const bf16* vt = ks + buf * LM_BN * LD;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int pair = warp + LM_WARPS * i;
      if (pair < n_pairs) {
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          o[2 * i + c][0] *= c0; o[2 * i + c][1] *= c0; o[2 * i + c][2] *= c1; o[2 * i + c][3] *= c1;
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          uint32_t b[4];
          lm_ldmatrix_x4_trans(b, vt + (kk * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * LD + pair * 16 + 8 * (lane >> 4));
          lm_mma(o[2 * i], pa[kk], b[0], b[1]);
          lm_mma(o[2 * i + 1], pa[kk], b[2], b[3]);
        }
      }
    }
    __syncthreads();   // everyone is done with this buffer, P and the maxima before they are overwritten
  }
  cp_async_wait<0>();
  if (n_splits == 1) {
    if (n_it == 0) return;
    float i0 = 1.0f / l0, i1 = 1.0f / l1;
    if (gate != nullptr) {
      if (h0 + r0 < n_head) i0 *= 1.0f / (1.0f + __expf(-gate[(size_t)t * ldg + h0 + r0]));
      if (h0 + r1 < n_head) i1 *= 1.0f / (1.0f + __expf(-gate[(size_t)t * ldg + h0 + r1]));
    }
#pragma unroll
    for (int i = 0; i < 2 * NP; ++i) {
      const int d = (warp + LM_WARPS * (i >> 1)) * 16 + (i & 1) * 8 + (lane & 3) * 2;
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        if (d + c < kv_rank) {
          if (h0 + r0 < n_head) out[(size_t)t * ldo + (size_t)(h0 + r0) * kv_rank + d + c] = from_float<bf16>(o[i][c] * i0);
          if (h0 + r1 < n_head) out[(size_t)t * ldo + (size_t)(h0 + r1) * kv_rank + d + c] = from_float<bf16>(o[i][2 + c] * i1);
        }
      }
    }
    return;
  }
  // ---- this piece's results where the other blocks of the cluster find them (the tiles' memory is free)
  if (n_it > 0) {
#pragma unroll
    for (int i = 0; i < 2 * NP; ++i) {
      const int d = (warp + LM_WARPS * (i >> 1)) * 16 + (i & 1) * 8 + (lane & 3) * 2;
#pragma unroll
      for (int c = 0; c < 2; ++c)
        if (d + c < kv_rank) {
          xo[r0 * kv_rank + d + c] = o[i][c];
          xo[r1 * kv_rank + d + c] = o[i][2 + c];
        }
    }
  }
  if (warp == 0 && (lane & 3) == 0) {
    stats[2 * r0] = m0; stats[2 * r0 + 1] = l0;
    stats[2 * r1] = m1; stats[2 * r1 + 1] = l1;
  }
  cluster_arrive();
  cluster_wait();
  for (int i = tid; i < n_splits * 2 * LM_HEADS; i += LM_WARPS * 32)
    all[i] = __uint_as_float(cluster_load(cluster_addr(stats + i % (2 * LM_HEADS), i / (2 * LM_HEADS))));
  __syncthreads();
  if (entry >= 0) {
    // every block merges its share of the (head, value) pairs
    for (int x = split * (LM_WARPS * 32) + tid; x < LM_HEADS * kv_rank; x += n_splits * (LM_WARPS * 32)) {
      const int hh = x / kv_rank, d = x % kv_rank;
      if (h0 + hh >= n_head) break;
      float M = -INFINITY;
      for (int sp = 0; sp < n_splits; ++sp) M = fmaxf(M, all[(sp * LM_HEADS + hh) * 2]);
      float L = 0.0f, acc = 0.0f;
      for (int sp = 0; sp < n_splits; ++sp) {
        const float ms = all[(sp * LM_HEADS + hh) * 2];
        if (ms == -INFINITY) continue;                     // an empty piece
        const float f = lm_pow2(ms - M);
        L += all[(sp * LM_HEADS + hh) * 2 + 1] * f;
        acc += __uint_as_float(cluster_load(cluster_addr(xo + x, sp))) * f;
      }
      float inv = 1.0f / L;
      if (gate != nullptr) inv *= 1.0f / (1.0f + __expf(-gate[(size_t)t * ldg + h0 + hh]));
      out[(size_t)t * ldo + (size_t)(h0 + hh) * kv_rank + d] = from_float<bf16>(acc * inv);
    }
  }
  __syncthreads();
  cluster_arrive();      // nobody leaves while its shared memory is read
  cluster_wait();
}

static size_t lm_smem_bytes(int D, int n_splits) {
  const size_t LD = ((D + 15) & ~15) + 8;
  return (LM_HEADS + 2 * LM_BN) * LD * 2 + (size_t)LM_HEADS * 72 * 2 +
         (2 * LM_WARPS * LM_HEADS + 2 * LM_HEADS + (size_t)n_splits * 2 * LM_HEADS) * 4;
}

template <int NP>
static int launch_latent_decode(const void* q, const void* cache, void* out, int ldo, const int* block_table, int max_blocks,
                                const int* rows, const int* row_entry, const int* positions, int n_rows, int n_head,
                                int kv_rank, int D, int page_size, int n_pages, float scale, int window, const float* gate,
                                int ldg, int* status, int n_splits, cudaStream_t stream) {
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_mma_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(latent_decode_mma_kernel<NP>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
    if (e != cudaSuccess) return (int)e;
    attr_set = true;
  }
  launch_pdl_cluster(latent_decode_mma_kernel<NP>, dim3(n_splits, (n_head + LM_HEADS - 1) / LM_HEADS, n_rows),
                     dim3(LM_WARPS * 32), lm_smem_bytes(D, n_splits), stream, n_splits, (const bf16*)q, (const bf16*)cache,
                     (bf16*)out, ldo, block_table, max_blocks, rows, row_entry, positions, n_head, kv_rank, D, page_size,
                     n_pages, scale, window, gate, ldg, status, n_splits);
  NIB_LAUNCH_CHECK();
}

}  // namespace nib

using namespace nib;

// 1 if the kernel takes these sizes: D a multiple of 8, kv_rank up to 512, the tiles within shared memory.
extern "C" int nib_latent_decode_mma_supported(int kv_rank, int D) {
  return D % 8 == 0 && kv_rank > 0 && kv_rank <= 512 && kv_rank <= D && lm_smem_bytes(D, LM_MAX_SPLITS) <= 200 * 1024 &&
         (size_t)LM_HEADS * kv_rank * 4 <= 2 * LM_BN * (size_t)(D + 8) * 2;
}

// q [T, n_head, D] contiguous bfloat16; cache: one layer [n_pages, page_size, D]; out [T, n_head * kv_rank].  rows: the
// step's rows to process (nullptr: rows 0..n_rows-1), single tokens.  n_splits (1, 2, 4, 8 or 16): the pieces of a row's
// keys, blocks of one cluster.
extern "C" int nib_latent_decode_mma(const void* q, const void* cache, void* out, int ldo, const int* block_table,
                                     int max_blocks, const int* rows, const int* row_entry, const int* positions, int n_rows,
                                     int n_head, int kv_rank, int D, int page_size, int n_pages, float scale, int window,
                                     const float* gate, int ldg, int* status, int n_splits, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (n_head <= 0 || page_size <= 0 ||
      !(n_splits == 1 || n_splits == 2 || n_splits == 4 || n_splits == 8 || n_splits == 16))
    return NIB_ERR_BAD_ARGUMENT;
  if (!nib_latent_decode_mma_supported(kv_rank, D) || n_rows > 65535) return NIB_ERR_UNSUPPORTED_SIZE;
  if (((uintptr_t)q & 15) || ((uintptr_t)cache & 15)) return NIB_ERR_UNSUPPORTED_SIZE;
#define NIB_LM(N)                                                                                                       \
  return launch_latent_decode<N>(q, cache, out, ldo, block_table, max_blocks, rows, row_entry, positions, n_rows, n_head, \
                                 kv_rank, D, page_size, n_pages, scale, window, gate, ldg, status, n_splits, stream)
  if (kv_rank <= 64) NIB_LM(1);
  if (kv_rank <= 128) NIB_LM(2);
  if (kv_rank <= 256) NIB_LM(4);
  NIB_LM(8);
#undef NIB_LM
}
