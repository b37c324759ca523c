// Attention for single decoded tokens in bfloat16, on warp-level MMAs whose rows are HEADS: the query heads that read the
// same cached rows are the rows of one MMA tile, so a tile of keys and values is read once from memory for all of them (up
// to sixteen a tile).  Two shapes of the cache:
//
//   keys and values in planes of their own, the query heads of a key/value head being its group (differential attention:
//   both maps of every head of the group, their queries laid into the row with zeros in the other map's place);
//   one plane whose row is key and value at once, all heads one group (a latent [c | k_rot], latent_attention.cu).
//
// One block takes a row, a tile of a group's heads and a piece of the row's keys.  Per tile of 64 keys: four warps make the
// scores of sixteen keys each (m16n8k16 over the key row), the row maxima and sums meet in shared memory, P lies there as
// bfloat16, and every warp adds P V for its share of the values.  Tiles come through two buffers by cp.async, the first of
// them ahead of griddepcontrol.wait where it does not hold the row's own key.  The pieces of a row are the blocks of one
// cluster: each leaves its (maximum, sum, unscaled result) in its own shared memory, and the warps of all of them share the
// merge through distributed shared memory, in the order of the pieces.  What is written:
//   a head's result, times sigmoid(gate[t, h]), or of a gate per element, where there is one; or (`diff`) for every pair of heads (2i, 2i + 1) the
//   difference a_2i - lambda a_2i+1 over its root mean square, times a constant (differential.cu says it for portions).
// With pooled blocks behind the window (one key and value for `pool` positions, rows of another list of pages of the same
// cache) a row's keys are one sequence, the blocks first; a learned sink joins the sum where the pieces merge.
// Scores (capped where asked for), softmax, sums, difference and norm are 32-bit.
#include "api.h"
#include "attention_extras.cuh"
#include "common.cuh"

namespace nib {

constexpr int GM_HEADS = 16, GM_BN = 64, GM_WARPS = 4, GM_THREADS = GM_WARPS * 32, GM_MAX_SPLITS = 16, GM_PLD = 72;

__device__ __forceinline__ void gm_ldmatrix_x4(uint32_t* r, const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void gm_ldmatrix_x4_trans(uint32_t* r, const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void gm_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float gm_pow2(float x) {   // the hardware's 2^x (relative error about 2^-22; 2^-inf = 0)
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float4 gm_cluster_load4(uint32_t addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
  return v;
}

struct GmParams {
  const bf16* q;
  int ldq;
  const bf16* cache;
  bf16* out;
  int ldo, out_head;            // rows and heads (or pairs of heads) of the result, in elements
  const int* block_table;
  int max_blocks;
  const int* rows;
  const int* row_entry;
  const int* positions;
  int n_head, n_kv_head, planes, row_dim, k_cols, v_cols, page_size, n_pages;
  float scale, softcap;
  int window;
  const float* gate;
  int ldg, gate_dim;            // gate_dim 0: one gate a head, else one for each of a head's first gate_dim values
  const float* sinks;           // a logit per head that joins the denominator (null: none)
  int pool;                     // > 0: blocks of so many positions behind the window are one key and value each,
  const int* pool_table;        // rows of these pages
  int diff;
  float lambda, eps, mul;
  int* status;
  int n_splits;
};

// NP: groups of sixteen values of the result that a warp owns (v_cols <= 64 NP)
template <int NP>
__global__ void __launch_bounds__(GM_THREADS)
attention_group_mma_kernel(const GmParams prm) {
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t gm_smem[];
  const bool shared_row = prm.planes == 1;
  const int Dk = (prm.k_cols + 15) & ~15, Dv = (prm.v_cols + 15) & ~15;
  const int LDK = Dk + 8, LDV = shared_row ? LDK : Dv + 8;            // rows padded against bank conflicts
  const int n_splits = prm.n_splits, v_cols = prm.v_cols, XR = (v_cols + 3) & ~3;
  bf16* qs = reinterpret_cast<bf16*>(gm_smem);                        // [16][LDK]
  bf16* ks = qs + GM_HEADS * LDK;                                     // [2][64][LDK]
  bf16* vs = shared_row ? ks : ks + 2 * GM_BN * LDK;                  // [2][64][LDV]
  bf16* ps = vs + 2 * GM_BN * LDV;                                    // [16][72]
  float* red = reinterpret_cast<float*>(ps + GM_HEADS * GM_PLD);      // [2][4 warps][16]
  float* stats = red + 2 * GM_WARPS * GM_HEADS;                       // [16][2]: this piece's maximum and sum
  float* all = stats + 2 * GM_HEADS;                                  // [splits][16][2]
  float* xo = reinterpret_cast<float*>(ks);                           // [16][XR], behind the last tile
  const int group = prm.n_head / prm.n_kv_head, m_tiles = (group + GM_HEADS - 1) / GM_HEADS;
  const int hk = blockIdx.y / m_tiles, h0 = hk * group + (blockIdx.y % m_tiles) * GM_HEADS;
  const int n_heads = min(GM_HEADS, (hk + 1) * group - h0);           // of this tile
  const int split = blockIdx.x;
  const int t = prm.rows ? prm.rows[blockIdx.z] : blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int entry = prm.row_entry[t], pos = prm.positions[t];
  // (a row of no request takes part in the cluster's barriers with an empty piece)
  const int lo = prm.window > 0 ? max(0, pos - prm.window + 1) : 0;
  // the row's keys in one sequence: its pooled blocks, then the window's positions (key k >= nb is position k + shift)
  const int nb = pooled_blocks_seen(pos, prm.window, prm.pool), shift = lo - nb, n_keys = pos + 1 - shift;
  const int per = ((n_keys - 1 + n_splits) / n_splits + 15) / 16 * 16;
  const int k_begin = split * per, k_end = entry < 0 ? 0 : min(n_keys, k_begin + per);
  const int n_it = k_end > k_begin ? (k_end - k_begin + GM_BN - 1) / GM_BN : 0;
  const int* table = prm.block_table + (size_t)max(entry, 0) * prm.max_blocks;
  const int* pool_table = prm.pool_table + (size_t)max(entry, 0) * prm.max_blocks;

  // the cached row (counted in rows of row_dim values) of key j for this group; -1: not there
  auto cached_row = [&](int k) -> int {
    if (k >= k_end) return -1;
    const int j = k < nb ? k : k + shift;
    const int page = (k < nb ? pool_table : table)[j / prm.page_size];
    if (page < 0 || page >= prm.n_pages) {
      *prm.status = NIB_STATUS_BAD_PAGE;
      return -1;
    }
    return (page * prm.planes * prm.n_kv_head + hk) * prm.page_size + j % prm.page_size;
  };
  // one plane of a tile: 64 rows of `pieces` (an even number) 16-byte pieces, of which those below `cols` values exist
  auto load_plane = [&](bf16* dst, int ld, int pieces, int cols, int row_lo, int row_hi, int plane_rows) {
    int r = tid / pieces, piece = tid % pieces;
    const int dr = GM_THREADS / pieces, dp = GM_THREADS % pieces;
    for (int i = 0; i < pieces / 2; ++i) {                            // 64 * pieces / 128 threads
      const int a = __shfl_sync(0xffffffffu, row_lo, r & 31), b = __shfl_sync(0xffffffffu, row_hi, r & 31);
      const int row = r < 32 ? a : b;
      const bool valid = row >= 0 && piece * 8 < cols;
      cp_async16(dst + r * ld + piece * 8,
                 valid ? prm.cache + (size_t)(row + plane_rows) * prm.row_dim + piece * 8 : prm.cache, valid);
      r += dr;
      piece += dp;
      if (piece >= pieces) {
        piece -= pieces;
        ++r;
      }
    }
  };
  auto load_tile = [&](int it, int buf) {
    const int j0 = k_begin + it * GM_BN;
    const int row_lo = cached_row(j0 + lane), row_hi = cached_row(j0 + 32 + lane);
    load_plane(ks + buf * GM_BN * LDK, LDK, Dk / 8, prm.row_dim, row_lo, row_hi, 0);
    if (!shared_row) load_plane(vs + buf * GM_BN * LDV, LDV, Dv / 8, prm.row_dim, row_lo, row_hi, prm.n_kv_head * prm.page_size);
  };
  const bool early = n_it > 0 && min(k_end, k_begin + GM_BN) < n_keys;  // the first tile does not hold the row's own key
  if (early) load_tile(0, 0);
  pdl_wait();
  if (n_it > 0) {
    const int pieces = Dk / 8;
    for (int c = tid; c < GM_HEADS * pieces; c += GM_THREADS) {
      const int r = c / pieces, piece = c % pieces;
      const bool valid = r < n_heads && piece * 8 < prm.row_dim;
      cp_async16(qs + r * LDK + piece * 8,
                 valid ? prm.q + (size_t)t * prm.ldq + (size_t)(h0 + r) * prm.row_dim + piece * 8 : prm.q, valid);
    }
    if (!early) load_tile(0, 0);
  }
  cp_async_commit();

  float o[2 * NP][4];
#pragma unroll
  for (int i = 0; i < 2 * NP; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;         // of heads lane / 4 and lane / 4 + 8 of the tile
  const int r0 = lane >> 2, r1 = r0 + 8, n_pairs = Dv / 16;
  constexpr float LOG2E = 1.4426950408889634f;
  const bool capped = prm.softcap > 0.0f;
  const float scale2 = prm.scale * LOG2E, cap2 = prm.softcap * LOG2E, cap_in = capped ? 2.0f * LOG2E * prm.scale / prm.softcap : 0.0f;
  for (int it = 0; it < n_it; ++it) {
    const int buf = it & 1;
    if (it + 1 < n_it) load_tile(it + 1, buf ^ 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    // ---- the scores of this warp's sixteen keys
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    const bf16* kt = ks + (buf * GM_BN + warp * 16) * LDK;
#pragma unroll 4
    for (int kk = 0; kk < Dk / 16; ++kk) {
      uint32_t a[4], b[4];
      gm_ldmatrix_x4(a, qs + ((lane & 7) + 8 * ((lane >> 3) & 1)) * LDK + kk * 16 + 8 * (lane >> 4));
      gm_ldmatrix_x4(b, kt + ((lane & 7) + 8 * (lane >> 4)) * LDK + kk * 16 + 8 * ((lane >> 3) & 1));
      gm_mma(s[0], a, b[0], b[1]);
      gm_mma(s[1], a, b[2], b[3]);
    }
    const int j_base = k_begin + it * GM_BN + warp * 16 + (lane & 3) * 2;
    float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        float v = s[i][c];
        // c tanh(x / c) by tanh(y) = 1 - 2 / (1 + e^2y) with the hardware's 2^x and division: relative error about 1e-6
        v = capped ? cap2 - __fdividef(2.0f * cap2, 1.0f + gm_pow2(v * cap_in)) : v * scale2;
        s[i][c] = j_base + i * 8 + (c & 1) < k_end ? v : -INFINITY;
        if (c < 2) mx0 = fmaxf(mx0, s[i][c]);
        else mx1 = fmaxf(mx1, s[i][c]);
      }
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    if ((lane & 3) == 0) {
      red[warp * GM_HEADS + r0] = mx0;
      red[warp * GM_HEADS + r1] = mx1;
    }
    __syncthreads();
    float n0 = m0, n1 = m1;
#pragma unroll
    for (int w = 0; w < GM_WARPS; ++w) {
      n0 = fmaxf(n0, red[w * GM_HEADS + r0]);
      n1 = fmaxf(n1, red[w * GM_HEADS + r1]);
    }
    // (every tile holds at least one live key: n0 and n1 are finite)
    float sum0 = 0.0f, sum1 = 0.0f;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        s[i][c] = gm_pow2(s[i][c] - n0);
        s[i][2 + c] = gm_pow2(s[i][2 + c] - n1);
        sum0 += s[i][c];
        sum1 += s[i][2 + c];
      }
      const int col = warp * 16 + i * 8 + (lane & 3) * 2;
      *reinterpret_cast<__nv_bfloat162*>(ps + r0 * GM_PLD + col) = __floats2bfloat162_rn(s[i][0], s[i][1]);
      *reinterpret_cast<__nv_bfloat162*>(ps + r1 * GM_PLD + col) = __floats2bfloat162_rn(s[i][2], s[i][3]);
    }
    sum0 += __shfl_xor_sync(0xffffffffu, sum0, 1);
    sum0 += __shfl_xor_sync(0xffffffffu, sum0, 2);
    sum1 += __shfl_xor_sync(0xffffffffu, sum1, 1);
    sum1 += __shfl_xor_sync(0xffffffffu, sum1, 2);
    float* sums = red + GM_WARPS * GM_HEADS;
    if ((lane & 3) == 0) {
      sums[warp * GM_HEADS + r0] = sum0;
      sums[warp * GM_HEADS + r1] = sum1;
    }
    __syncthreads();
    const float c0 = gm_pow2(m0 - n0), c1 = gm_pow2(m1 - n1);          // (2^-inf = 0 at the first tile)
    l0 *= c0;
    l1 *= c1;
#pragma unroll
    for (int w = 0; w < GM_WARPS; ++w) {
      l0 += sums[w * GM_HEADS + r0];
      l1 += sums[w * GM_HEADS + r1];
    }
    m0 = n0;
    m1 = n1;
    // ---- O += P V for this warp's values: groups warp, warp + 4, ... of sixteen
    uint32_t pa[4][4];
#pragma unroll
    for (int kk = 0; kk < 4; ++kk)
      gm_ldmatrix_x4(pa[kk], ps + ((lane & 7) + 8 * ((lane >> 3) & 1)) * GM_PLD + kk * 16 + 8 * (lane >> 4));
    const bf16* vt = vs + buf * GM_BN * LDV;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int pair = warp + GM_WARPS * i;
      if (pair < n_pairs) {
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          o[2 * i + c][0] *= c0; o[2 * i + c][1] *= c0; o[2 * i + c][2] *= c1; o[2 * i + c][3] *= c1;
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          uint32_t b[4];
          gm_ldmatrix_x4_trans(b, vt + (kk * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * LDV + pair * 16 + 8 * (lane >> 4));
          gm_mma(o[2 * i], pa[kk], b[0], b[1]);
          gm_mma(o[2 * i + 1], pa[kk], b[2], b[3]);
        }
      }
    }
    __syncthreads();   // everyone is done with this buffer, P and the maxima before they are overwritten
  }
  cp_async_wait<0>();
  // ---- this piece's results where the blocks of the cluster find them (the tiles' memory is free)
  if (n_it > 0) {
#pragma unroll
    for (int i = 0; i < 2 * NP; ++i) {
      const int d = (warp + GM_WARPS * (i >> 1)) * 16 + (i & 1) * 8 + (lane & 3) * 2;
#pragma unroll
      for (int c = 0; c < 2; ++c)
        if (d + c < XR) {
          xo[r0 * XR + d + c] = o[i][c];
          xo[r1 * XR + d + c] = o[i][2 + c];
        }
    }
  }
  if (warp == 0 && (lane & 3) == 0) {
    stats[2 * r0] = m0; stats[2 * r0 + 1] = l0;
    stats[2 * r1] = m1; stats[2 * r1 + 1] = l1;
  }
  if (n_splits > 1) {
    cluster_arrive();
    cluster_wait();
    for (int i = tid; i < n_splits * 2 * GM_HEADS; i += GM_THREADS)
      all[i] = __uint_as_float(cluster_load(cluster_addr(stats + i % (2 * GM_HEADS), i / (2 * GM_HEADS))));
  } else {
    __syncthreads();
    for (int i = tid; i < 2 * GM_HEADS; i += GM_THREADS) all[i] = stats[i];
  }
  __syncthreads();
  if (entry >= 0) {
    // head hh's values d .. d + 3 out of all pieces, divided by the softmax's sum
    auto merged4 = [&](int hh, int d) -> float4 {
      float M = -INFINITY;
      for (int sp = 0; sp < n_splits; ++sp) M = fmaxf(M, all[(sp * GM_HEADS + hh) * 2]);
      float L = 0.0f;
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int s0 = 0; s0 < n_splits; s0 += 8) {
        float4 x[8];
#pragma unroll
        for (int i = 0; i < 8; ++i)                        // (asked for together: each is a trip to another SM)
          if (s0 + i < n_splits)
            x[i] = n_splits > 1 ? gm_cluster_load4(cluster_addr(xo + hh * XR + d, s0 + i)) : *reinterpret_cast<const float4*>(xo + hh * XR + d);
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (s0 + i < n_splits) {
            const float ms = all[((s0 + i) * GM_HEADS + hh) * 2];
            if (ms != -INFINITY) {                         // (an empty piece left nothing)
              const float f = gm_pow2(ms - M);
              L += all[((s0 + i) * GM_HEADS + hh) * 2 + 1] * f;
              acc.x += x[i].x * f; acc.y += x[i].y * f; acc.z += x[i].z * f; acc.w += x[i].w * f;
            }
          }
      }
      if (prm.sinks != nullptr) L += gm_pow2(prm.sinks[h0 + hh] * LOG2E - M);
      const float inv = 1.0f / L;
      return make_float4(acc.x * inv, acc.y * inv, acc.z * inv, acc.w * inv);
    };
    const int me = split * GM_WARPS + warp, n_warps = n_splits * GM_WARPS;
    bf16* row = prm.out + (size_t)t * prm.ldo;
    if (!prm.diff) {
      const int parts = (v_cols + 127) / 128;              // a warp takes 128 values of a head at a time
      for (int u = me; u < n_heads * parts; u += n_warps) {
        const int hh = u / parts, d = (u % parts) * 128 + 4 * lane;
        if (d >= v_cols) continue;
        const float4 v = merged4(hh, d);
        const float g = prm.gate && prm.gate_dim == 0 ? 1.0f / (1.0f + __expf(-prm.gate[(size_t)t * prm.ldg + h0 + hh])) : 1.0f;
        bf16* dst = row + (size_t)(h0 + hh) * prm.out_head + d;
        float w[4] = {v.x * g, v.y * g, v.z * g, v.w * g};
        if (prm.gate_dim > 0) {
          const float* gr = prm.gate + (size_t)t * prm.ldg + (size_t)(h0 + hh) * prm.gate_dim + d;
#pragma unroll
          for (int c = 0; c < 4; ++c)
            if (d + c < prm.gate_dim) w[c] *= 1.0f / (1.0f + __expf(-gr[c]));
        }
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (d + c < v_cols) dst[c] = from_float<bf16>(w[c]);
      }
    } else {
      for (int u = me; u < n_heads / 2; u += n_warps) {
        float w[2][4], q = 0.0f;                           // v_cols <= 256: two pieces of four values a lane
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int d = i * 128 + 4 * lane;
          w[i][0] = w[i][1] = w[i][2] = w[i][3] = 0.0f;
          if (d < v_cols) {
            const float4 a1 = merged4(2 * u, d), a2 = merged4(2 * u + 1, d);
            w[i][0] = fmaf(-prm.lambda, a2.x, a1.x);
            w[i][1] = d + 1 < v_cols ? fmaf(-prm.lambda, a2.y, a1.y) : 0.0f;
            w[i][2] = d + 2 < v_cols ? fmaf(-prm.lambda, a2.z, a1.z) : 0.0f;
            w[i][3] = d + 3 < v_cols ? fmaf(-prm.lambda, a2.w, a1.w) : 0.0f;
          }
          q += w[i][0] * w[i][0] + w[i][1] * w[i][1] + w[i][2] * w[i][2] + w[i][3] * w[i][3];
        }
        const float f = prm.mul / sqrtf(warp_sum(q) / (float)v_cols + prm.eps);
        bf16* dst = row + (size_t)(h0 / 2 + u) * prm.out_head;
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const int d = i * 128 + 4 * lane + c;
            if (d < v_cols) dst[d] = from_float<bf16>(w[i][c] * f);
          }
      }
    }
  }
  if (n_splits > 1) {      // nobody leaves while its shared memory is read
    __syncthreads();
    cluster_arrive();
    cluster_wait();
  }
}

static size_t gm_smem_bytes(int planes, int k_cols, int v_cols, int n_splits) {
  const size_t LDK = ((k_cols + 15) & ~15) + 8, LDV = planes == 1 ? 0 : ((v_cols + 15) & ~15) + 8;
  return (GM_HEADS * LDK + 2 * GM_BN * (LDK + LDV)) * 2 + (size_t)GM_HEADS * GM_PLD * 2 +
         (2 * GM_WARPS * GM_HEADS + 2 * GM_HEADS + (size_t)n_splits * 2 * GM_HEADS) * 4;
}

template <int NP>
static int launch_group_mma(const GmParams& prm, int n_rows, cudaStream_t stream) {
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(attention_group_mma_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(attention_group_mma_kernel<NP>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
    if (e != cudaSuccess) return (int)e;
    attr_set = true;
  }
  const int group = prm.n_head / prm.n_kv_head, m_tiles = (group + GM_HEADS - 1) / GM_HEADS;
  launch_pdl_cluster(attention_group_mma_kernel<NP>, dim3(prm.n_splits, prm.n_kv_head * m_tiles, n_rows), dim3(GM_THREADS),
                     gm_smem_bytes(prm.planes, prm.k_cols, prm.v_cols, prm.n_splits), stream, prm.n_splits, prm);
  NIB_LAUNCH_CHECK();
}

}  // namespace nib

using namespace nib;

// 1 if the kernel takes these sizes: rows of a multiple of 8 values (16 with planes of their own), v_cols up to 512 (256 for
// differences of pairs), the tiles within shared memory.  k_cols: the values of a key row that count, from its start.
extern "C" int nib_attention_group_mma_supported(int row_dim, int planes, int k_cols, int v_cols, int diff) {
  if (row_dim <= 0 || (planes != 1 && planes != 2) || row_dim % (planes == 1 ? 8 : 16)) return 0;
  if (k_cols <= 0 || k_cols > row_dim || v_cols <= 0 || v_cols > row_dim || v_cols > (diff ? 256 : 512)) return 0;
  if (planes == 1 && k_cols != row_dim) return 0;
  return gm_smem_bytes(planes, k_cols, v_cols, GM_MAX_SPLITS) <= 220 * 1024;
}

// q [T rows, ldq], heads of row_dim values one after the other; cache: one layer [n_pages, planes, n_kv_head, page_size,
// row_dim].  rows: the step's rows to process (nullptr: rows 0..n_rows-1), single tokens.  n_splits (1, 2, 4, 8 or 16): the
// pieces of a row's keys, blocks of one cluster.
extern "C" int nib_attention_group_mma(const void* q, int ldq, const void* cache, int planes, void* out, int ldo, int out_head,
                                       const int* block_table, int max_blocks, const int* rows, const int* row_entry,
                                       const int* positions, int n_rows, int n_head, int n_kv_head, int row_dim, int k_cols,
                                       int v_cols, int page_size, int n_pages, float scale, int window, float softcap,
                                       const float* gate, int ldg, int gate_dim, const float* sinks, int pool, const int* pool_table,
                                       int diff, float lambda, float eps, float mul, int* status,
                                       int n_splits, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (n_head <= 0 || n_kv_head <= 0 || n_head % n_kv_head || page_size <= 0 || softcap < 0.0f ||
      !(n_splits == 1 || n_splits == 2 || n_splits == 4 || n_splits == 8 || n_splits == 16))
    return NIB_ERR_BAD_ARGUMENT;
  if (diff && (n_head / n_kv_head) % 2) return NIB_ERR_BAD_ARGUMENT;
  if (pool < 0 || gate_dim < 0 || (pool > 0 && (window <= 0 || pool_table == nullptr)) || (gate_dim > 0 && gate == nullptr))
    return NIB_ERR_BAD_ARGUMENT;
  if (!nib_attention_group_mma_supported(row_dim, planes, k_cols, v_cols, diff) || n_rows > 65535) return NIB_ERR_UNSUPPORTED_SIZE;
  if (((uintptr_t)q & 15) || ((uintptr_t)cache & 15) || (ldq & 7)) return NIB_ERR_UNSUPPORTED_SIZE;
  if ((long long)n_pages * planes * n_kv_head * page_size > 0x7fffffffll) return NIB_ERR_UNSUPPORTED_SIZE;
  GmParams prm;
  prm.q = (const bf16*)q; prm.ldq = ldq; prm.cache = (const bf16*)cache; prm.out = (bf16*)out; prm.ldo = ldo;
  prm.out_head = out_head; prm.block_table = block_table; prm.max_blocks = max_blocks; prm.rows = rows;
  prm.row_entry = row_entry; prm.positions = positions; prm.n_head = n_head; prm.n_kv_head = n_kv_head; prm.planes = planes;
  prm.row_dim = row_dim; prm.k_cols = k_cols; prm.v_cols = v_cols; prm.page_size = page_size; prm.n_pages = n_pages;
  prm.scale = scale; prm.softcap = softcap; prm.window = window; prm.gate = gate; prm.ldg = ldg; prm.diff = diff;
  prm.gate_dim = gate_dim; prm.sinks = sinks; prm.pool = pool; prm.pool_table = pool > 0 ? pool_table : block_table;
  prm.lambda = lambda; prm.eps = eps; prm.mul = mul; prm.status = status; prm.n_splits = n_splits;
  if (v_cols <= 64) return launch_group_mma<1>(prm, n_rows, stream);
  if (v_cols <= 128) return launch_group_mma<2>(prm, n_rows, stream);
  if (v_cols <= 256) return launch_group_mma<4>(prm, n_rows, stream);
  return launch_group_mma<8>(prm, n_rows, stream);
}
