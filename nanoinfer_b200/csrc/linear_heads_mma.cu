// The product per head of linear_heads.cu on warp-level MMAs (bfloat16 operands, 32-bit sums):
//   out[t, h, :N] = a[t, h, :K] . w[h]^T,   w [H, N, K],   out bfloat16 or float32,
// times sigmoid(gate[t, h, n]) where there is a gate (32-bit logits),
// and, where the heads of `a` hold a rotated part behind the K values (a latent attention's queries [K unrotated | rot_dim
// rotated]), that part turned by the row's position and written behind the N values of the same head in the same launch:
// the query of a head over a shared latent.
//
// A block owns a tile of rows x 64 columns of one head; K is walked in pieces of 64 through two buffers by cp.async.  Steps
// of many rows: 64 rows a block, sixteen a warp; steps of at most 16 rows: all rows in every warp, sixteen columns a warp.
#include "api.h"
#include "common.cuh"

namespace nib {

constexpr int LH_BN = 64, LH_KC = 64, LH_LD = LH_KC + 8;

__device__ __forceinline__ void lh_ldmatrix_x4(uint32_t* r, const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void lh_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct RotTail {
  const int* positions;
  const double* freqs;
  int rot_dim, rot_dims, halves;
};

template <int BM, typename OutT>
__global__ void __launch_bounds__(128)
linear_heads_mma_kernel(const bf16* a, int lda, int a_hs, const bf16* __restrict__ w, OutT* out, int ldo, int o_hs, int M,
                        int N, int K, RotTail rot, const float* gate, int ldg) {
  pdl_trigger();
  __shared__ __align__(16) bf16 as[2][BM * LH_LD];
  __shared__ __align__(16) bf16 ws[2][LH_BN * LH_LD];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n0 = blockIdx.x * LH_BN, m0 = blockIdx.y * BM, h = blockIdx.z;
  if (n0 >= N) {
    // ---- the head's rotated part of this tile's rows, a thread a (row, pair or passing value)
    const int half = rot.rot_dims / 2, per_row = half + (rot.rot_dim - rot.rot_dims);
    const int rows = min(BM, M - m0);
    pdl_wait();
    for (int x = tid; x < rows * per_row; x += 128) {
      const int m = m0 + x / per_row, i = x % per_row;
      const bf16* src = a + (size_t)m * lda + (size_t)h * a_hs + K;
      OutT* dst = out + (size_t)m * ldo + (size_t)h * o_hs + N;
      if (i < half) {
        double sd, cd;
        sincos((double)rot.positions[m] * rot.freqs[i], &sd, &cd);
        const float c = (float)cd, s = (float)sd;
        const int iu = rot.halves ? i : 2 * i, iv = rot.halves ? i + half : 2 * i + 1;
        const float u = to_float(src[iu]), v = to_float(src[iv]);
        dst[iu] = from_float<OutT>(u * c - v * s);
        dst[iv] = from_float<OutT>(v * c + u * s);
      } else {
        const int d = rot.rot_dims + (i - half);
        dst[d] = from_float<OutT>(to_float(src[d]));
      }
    }
    return;
  }
  constexpr int NT = BM == 64 ? 8 : 2;                      // 8-column tiles of a warp
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
  const bf16* wh = w + (size_t)h * N * K;
  auto load_w = [&](int k0, int buf) {
    for (int c = tid; c < LH_BN * (LH_KC / 8); c += 128) {
      const int r = c >> 3, k = k0 + (c & 7) * 8;
      const bool valid = n0 + r < N && k < K;
      cp_async16(&ws[buf][r * LH_LD + (c & 7) * 8], valid ? wh + (size_t)(n0 + r) * K + k : wh, valid);
    }
  };
  auto load_a = [&](int k0, int buf) {
    for (int c = tid; c < BM * (LH_KC / 8); c += 128) {
      const int r = c >> 3, k = k0 + (c & 7) * 8;
      const bool valid = m0 + r < M && k < K;
      cp_async16(&as[buf][r * LH_LD + (c & 7) * 8], valid ? a + (size_t)(m0 + r) * lda + (size_t)h * a_hs + k : a, valid);
    }
  };
  load_w(0, 0);                                             // (weights do not wait for the kernel ahead)
  pdl_wait();
  load_a(0, 0);
  cp_async_commit();
  const int n_k = (K + LH_KC - 1) / LH_KC;
  float gates[NT][4];                                       // (asked for here, they travel while the products are made)
  if (gate != nullptr) {
    const int ga = m0 + (BM == 64 ? warp * 16 : 0) + (lane >> 2), gc = n0 + (BM == 64 ? 0 : warp * 16) + (lane & 3) * 2;
    const bool pairs = ((uintptr_t)gate & 7) == 0 && (ldg & 1) == 0 && (N & 1) == 0;
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int c = 0; c < 4; c += 2) {
        const int m = ga + (c < 2 ? 0 : 8), col = gc + i * 8;
        const float* g = gate + (size_t)m * ldg + (size_t)h * N + col;
        gates[i][c] = gates[i][c + 1] = 0.0f;
        if (m < M && col < N) {
          if (pairs) {
            const float2 v = *reinterpret_cast<const float2*>(g);
            gates[i][c] = v.x;
            gates[i][c + 1] = v.y;
          } else {
            gates[i][c] = g[0];
            if (col + 1 < N) gates[i][c + 1] = g[1];
          }
        }
      }
  }
  const int arow = BM == 64 ? warp * 16 : 0, bcol = BM == 64 ? 0 : warp * 16;
  for (int kc = 0; kc < n_k; ++kc) {
    const int buf = kc & 1;
    if (kc + 1 < n_k) {
      load_w((kc + 1) * LH_KC, buf ^ 1);
      load_a((kc + 1) * LH_KC, buf ^ 1);
    }
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < LH_KC / 16; ++kk) {
      uint32_t af[4];
      lh_ldmatrix_x4(af, &as[buf][(arow + (lane & 7) + 8 * ((lane >> 3) & 1)) * LH_LD + kk * 16 + 8 * (lane >> 4)]);
#pragma unroll
      for (int nn = 0; nn < NT / 2; ++nn) {
        uint32_t b[4];
        lh_ldmatrix_x4(b, &ws[buf][(bcol + nn * 16 + (lane & 7) + 8 * (lane >> 4)) * LH_LD + kk * 16 + 8 * ((lane >> 3) & 1)]);
        lh_mma(acc[2 * nn], af, b[0], b[1]);
        lh_mma(acc[2 * nn + 1], af, b[2], b[3]);
      }
    }
    __syncthreads();
  }
  const int ra = m0 + arow + (lane >> 2), rb = ra + 8;
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    const int n = n0 + bcol + i * 8 + (lane & 3) * 2;
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int m = c < 2 ? ra : rb, col = n + (c & 1);
      if (m >= M || col >= N) continue;
      const float y = gate ? acc[i][c] / (1.0f + __expf(-gates[i][c])) : acc[i][c];
      out[(size_t)m * ldo + (size_t)h * o_hs + col] = from_float<OutT>(y);
    }
  }
}

template <typename OutT>
static int launch_linear_heads_mma(const void* a, int lda, int a_hs, const void* w, void* out, int ldo, int o_hs, int M,
                                   int n_head, int N, int K, RotTail rot, const float* gate, int ldg, cudaStream_t stream) {
  const int nb = (N + LH_BN - 1) / LH_BN + (rot.rot_dim > 0 ? 1 : 0);
  if (M <= 16)
    launch_pdl(linear_heads_mma_kernel<16, OutT>, dim3(nb, (M + 15) / 16, n_head), dim3(128), 0, stream, (const bf16*)a, lda,
               a_hs, (const bf16*)w, (OutT*)out, ldo, o_hs, M, N, K, rot, gate, ldg);
  else
    launch_pdl(linear_heads_mma_kernel<64, OutT>, dim3(nb, (M + 63) / 64, n_head), dim3(128), 0, stream, (const bf16*)a, lda,
               a_hs, (const bf16*)w, (OutT*)out, ldo, o_hs, M, N, K, rot, gate, ldg);
  NIB_LAUNCH_CHECK();
}

}  // namespace nib

using namespace nib;

// 1 if the MMA form takes these operands: K, the row pitch and the heads' stride multiples of 8, 16-byte aligned pointers.
extern "C" int nib_linear_heads_mma_supported(const void* a, int lda, int a_head_stride, const void* w, int K) {
  return K > 0 && (K & 7) == 0 && (lda & 7) == 0 && (a_head_stride & 7) == 0 && ((uintptr_t)a & 15) == 0 &&
         ((uintptr_t)w & 15) == 0;
}

// rot_dim > 0: a's heads are [K | rot_dim] and out's heads [N | rot_dim]; the rotated part (pairs (2i, 2i + 1) of its first
// rot_dims values, or halves) goes behind the product's N values.
extern "C" int nib_linear_heads_mma(int out_dtype, const void* a, int lda, int a_head_stride, const void* w, void* out,
                                    int ldo, int out_head_stride, int M, int n_head, int N, int K, const int* positions,
                                    const double* freqs, int rot_dim, int rot_dims, int halves, const float* gate,
                                    int ldg, cudaStream_t stream) {
  if (M <= 0 || n_head <= 0 || N <= 0) return 0;
  if (!nib_linear_heads_mma_supported(a, lda, a_head_stride, w, K)) return NIB_ERR_UNSUPPORTED_SIZE;
  if (rot_dim < 0 || rot_dims < 0 || rot_dims > rot_dim || (rot_dims & 1) || (rot_dims > 0 && freqs == nullptr) ||
      (rot_dim > 0 && positions == nullptr))
    return NIB_ERR_BAD_ARGUMENT;
  if ((M + 15) / 16 > 65535 || n_head > 65535) return NIB_ERR_UNSUPPORTED_SIZE;
  const RotTail rot = {positions, freqs, rot_dim, rot_dims, halves};
  if (out_dtype == DT_F32)
    return launch_linear_heads_mma<float>(a, lda, a_head_stride, w, out, ldo, out_head_stride, M, n_head, N, K, rot, gate, ldg, stream);
  if (out_dtype == DT_BF16)
    return launch_linear_heads_mma<bf16>(a, lda, a_head_stride, w, out, ldo, out_head_stride, M, n_head, N, K, rot, gate, ldg, stream);
  return NIB_ERR_BAD_ARGUMENT;
}
