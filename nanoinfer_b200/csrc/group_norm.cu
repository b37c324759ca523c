// Norms in groups on the 32-bit residual stream: a row of C values is cut into `groups` equal consecutive parts, each
// part is divided by its own root mean square (eps inside the root), and the whole row is multiplied by w.
//
//   group_norm       : v = x[rows[r]] (+ add); out[r] = norm(v); with `add`, one vector for all rows, v is also written
//                      back to x: a looped stack of layers adds such a vector to the stream ahead of each pass, in the
//                      norm that the pass's first layer starts with; `add_rows` is a row of its own for each row, added
//                      ahead of the vector (the embedding's output, given to every later pass again).  Without `out` only the sum is made.
//   embed_group_norm : x[t] = norm(table[token_t] * scale): the embedding and the norm that follows it in one pass.
//
// A warp owns a (row, part): parts do not see one another, so there is no shared memory and no block barrier (one group and
// at most 64 rows: a block a row).  Parts
// whose size is a multiple of 4 (up to 2048) live in registers as 16-byte pieces; others are read twice.
#include "api.h"
#include "common.cuh"

namespace nib {

__device__ __forceinline__ void gn_store4(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
__device__ __forceinline__ void gn_store4(bf16* p, float a, float b, float c, float d) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
  uint2 u;
  u.x = *reinterpret_cast<uint32_t*>(&lo);
  u.y = *reinterpret_cast<uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = u;
}
__device__ __forceinline__ float4 gn_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 gn_load4(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}

// Where a row comes from: the stream (optionally through a list of rows, optionally with a vector added), or a table
// looked up by token.
template <typename T>
struct StreamSource {
  static constexpr bool WRITES_BACK = true;
  float* x;
  const int* rows;
  const float* add;
  const float* add_rows;           // more rows [., C] to add, one a row of the stream (null: none)
  __device__ __forceinline__ bool adds() const { return add != nullptr || add_rows != nullptr; }
  __device__ __forceinline__ float* row(int r, int C) const { return x + (size_t)(rows ? rows[r] : r) * C; }
};
template <typename T>
struct TableSource {
  static constexpr bool WRITES_BACK = false;
  const int* tokens;
  const int* feedback;
  const T* table;
  float scale;
  __device__ __forceinline__ const T* row(int r, int C) const {
    int tok = tokens[r];
    if (tok < 0) tok = feedback[-tok - 1];   // the token that the step before sampled for slot -tok - 1
    return table + (size_t)tok * C;
  }
};

template <typename Src, typename OutT, int NV>
__global__ void __launch_bounds__(256)
group_norm_vec_kernel(Src src, const float* __restrict__ w, OutT* out, int n_rows, int C, int groups, float eps) {
  pdl_trigger();
  const int lane = threadIdx.x & 31;
  const int unit = blockIdx.x * 8 + (threadIdx.x >> 5);
  const int r = unit / groups, g = unit % groups;
  const int gs = C / groups, n4 = gs >> 2, c0 = g * gs;
  float4 ww[NV];                                   // (the weights do not wait for the kernel ahead)
  if (out != nullptr) {
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (lane + 32 * i < n4) ww[i] = gn_load4(w + c0 + 4 * (lane + 32 * i));
  }
  pdl_wait();
  if (r >= n_rows) return;
  auto* p = src.row(r, C) + c0;
  float4 v[NV];
  float q = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int k = lane + 32 * i;
    if (k < n4) {
      v[i] = gn_load4(p + 4 * k);
      if constexpr (Src::WRITES_BACK) {
        if (src.add_rows != nullptr) {
          const float4 b = gn_load4(src.add_rows + (size_t)r * C + c0 + 4 * k);
          v[i] = make_float4(v[i].x + b.x, v[i].y + b.y, v[i].z + b.z, v[i].w + b.w);
        }
        if (src.add != nullptr) {
          const float4 a = gn_load4(src.add + c0 + 4 * k);
          v[i] = make_float4(v[i].x + a.x, v[i].y + a.y, v[i].z + a.z, v[i].w + a.w);
        }
        if (src.adds()) gn_store4(p + 4 * k, v[i].x, v[i].y, v[i].z, v[i].w);
      } else {
        v[i] = make_float4(v[i].x * src.scale, v[i].y * src.scale, v[i].z * src.scale, v[i].w * src.scale);
      }
      q += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
  }
  if (out == nullptr) return;
  const float rstd = 1.0f / sqrtf(warp_sum(q) / (float)gs + eps);
  OutT* o = out + (size_t)r * C + c0;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int k = lane + 32 * i;
    if (k < n4) {
      gn_store4(o + 4 * k, v[i].x * rstd * ww[i].x, v[i].y * rstd * ww[i].y, v[i].z * rstd * ww[i].z, v[i].w * rstd * ww[i].w);
    }
  }
}

// The same with one group and a block a row, a 16-byte piece a thread: steps of few rows, where a warp's row is a chain of
// loads and stores that nothing else fills.
template <typename Src, typename OutT, int NV>
__global__ void __launch_bounds__(256)
group_norm_row_kernel(Src src, const float* __restrict__ w, OutT* out, int n_rows, int C, float eps) {
  pdl_trigger();
  __shared__ float sums[32];
  const int r = blockIdx.x, n4 = C >> 2;
  float4 ww[NV];
  if (out != nullptr) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int k = threadIdx.x + blockDim.x * i;
      if (k < n4) ww[i] = gn_load4(w + 4 * k);
    }
  }
  pdl_wait();
  auto* p = src.row(r, C);
  float4 v[NV];
  float q = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int k = threadIdx.x + blockDim.x * i;
    if (k < n4) {
      v[i] = gn_load4(p + 4 * k);
      if constexpr (Src::WRITES_BACK) {
        if (src.add_rows != nullptr) {
          const float4 b = gn_load4(src.add_rows + (size_t)r * C + 4 * k);
          v[i] = make_float4(v[i].x + b.x, v[i].y + b.y, v[i].z + b.z, v[i].w + b.w);
        }
        if (src.add != nullptr) {
          const float4 a = gn_load4(src.add + 4 * k);
          v[i] = make_float4(v[i].x + a.x, v[i].y + a.y, v[i].z + a.z, v[i].w + a.w);
        }
        if (src.adds()) gn_store4(p + 4 * k, v[i].x, v[i].y, v[i].z, v[i].w);
      } else {
        v[i] = make_float4(v[i].x * src.scale, v[i].y * src.scale, v[i].z * src.scale, v[i].w * src.scale);
      }
      q += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
  }
  if (out == nullptr) return;
  const float rstd = 1.0f / sqrtf(block_sum(q, sums) / (float)C + eps);
  OutT* o = out + (size_t)r * C;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int k = threadIdx.x + blockDim.x * i;
    if (k < n4)
      gn_store4(o + 4 * k, v[i].x * rstd * ww[i].x, v[i].y * rstd * ww[i].y, v[i].z * rstd * ww[i].z, v[i].w * rstd * ww[i].w);
  }
}

template <typename Src, typename OutT>
__global__ void __launch_bounds__(256)
group_norm_any_kernel(Src src, const float* __restrict__ w, OutT* out, int n_rows, int C, int groups, float eps) {
  pdl_trigger();
  const int lane = threadIdx.x & 31;
  const int unit = blockIdx.x * 8 + (threadIdx.x >> 5);
  const int r = unit / groups, g = unit % groups;
  const int gs = C / groups, c0 = g * gs;
  pdl_wait();
  if (r >= n_rows) return;
  auto* p = src.row(r, C) + c0;
  float q = 0.0f;
  for (int c = lane; c < gs; c += 32) {
    float v = to_float(p[c]);
    if constexpr (Src::WRITES_BACK) {
      if (src.add_rows != nullptr) v += src.add_rows[(size_t)r * C + c0 + c];
      if (src.add != nullptr) v += src.add[c0 + c];
      if (src.adds()) p[c] = v;
    } else {
      v *= src.scale;
    }
    q += v * v;
  }
  if (out == nullptr) return;
  const float rstd = 1.0f / sqrtf(warp_sum(q) / (float)gs + eps);
  OutT* o = out + (size_t)r * C + c0;
  for (int c = lane; c < gs; c += 32) {      // (a lane reads again what it read, or wrote, itself)
    float v = to_float(p[c]);
    if constexpr (!Src::WRITES_BACK) v *= src.scale;
    o[c] = from_float<OutT>(v * rstd * w[c0 + c]);
  }
}

template <typename Src, typename OutT>
static int launch_group_norm(Src src, bool aligned, const float* w, OutT* out, int n_rows, int C, int groups, float eps,
                             cudaStream_t stream) {
  const int gs = C / groups;
  const long long units = (long long)n_rows * groups;
  const dim3 grid((unsigned)((units + 7) / 8));
  const bool vec = aligned && (gs & 3) == 0 && gs <= 2048 && (((uintptr_t)w | (uintptr_t)out) & 15) == 0;
  if (vec && groups == 1 && C >= 256 && n_rows <= 64) {
    const int n4 = C >> 2, threads = n4 >= 256 ? 256 : (n4 + 31) / 32 * 32;
    if (n4 <= 256) launch_pdl(group_norm_row_kernel<Src, OutT, 1>, dim3(n_rows), dim3(threads), 0, stream, src, w, out, n_rows, C, eps);
    else launch_pdl(group_norm_row_kernel<Src, OutT, 2>, dim3(n_rows), dim3(threads), 0, stream, src, w, out, n_rows, C, eps);
    NIB_LAUNCH_CHECK();
  }
#define NIB_GN(NV) launch_pdl(group_norm_vec_kernel<Src, OutT, NV>, grid, dim3(256), 0, stream, src, w, out, n_rows, C, groups, eps)
  if (vec && gs <= 256) NIB_GN(2);
  else if (vec && gs <= 512) NIB_GN(4);
  else if (vec && gs <= 1024) NIB_GN(8);
  else if (vec) NIB_GN(16);
  else launch_pdl(group_norm_any_kernel<Src, OutT>, grid, dim3(256), 0, stream, src, w, out, n_rows, C, groups, eps);
#undef NIB_GN
  NIB_LAUNCH_CHECK();
}

}  // namespace nib

using namespace nib;

extern "C" int nib_group_norm(int out_dtype, float* x, const int* rows, const float* add, const float* add_rows, const float* w, void* out,
                              int n_rows, int C, int groups, float eps, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (C <= 0 || groups <= 0 || C % groups != 0 || ((add != nullptr || add_rows != nullptr) && rows != nullptr) ||
      (out == nullptr && add == nullptr && add_rows == nullptr) ||
      (out != nullptr && w == nullptr))
    return NIB_ERR_BAD_ARGUMENT;
  const bool aligned = (((uintptr_t)x | (uintptr_t)add | (uintptr_t)add_rows) & 15) == 0;
  if (out_dtype == DT_F32)
    return launch_group_norm(StreamSource<float>{x, rows, add, add_rows}, aligned, w, (float*)out, n_rows, C, groups, eps, stream);
  if (out_dtype == DT_BF16)
    return launch_group_norm(StreamSource<float>{x, rows, add, add_rows}, aligned, w, (bf16*)out, n_rows, C, groups, eps, stream);
  return NIB_ERR_BAD_ARGUMENT;
}

extern "C" int nib_embed_group_norm(int dtype, const int* tokens, const int* feedback, const void* table, float scale,
                                    const float* w, float* x, int T, int C, int groups, float eps, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (C <= 0 || groups <= 0 || C % groups != 0) return NIB_ERR_BAD_ARGUMENT;
  const bool aligned = ((uintptr_t)table & 15) == 0;
  if (dtype == DT_F32)
    return launch_group_norm(TableSource<float>{tokens, feedback, (const float*)table, scale}, aligned, w, x, T, C, groups,
                             eps, stream);
  if (dtype == DT_BF16)
    return launch_group_norm(TableSource<bf16>{tokens, feedback, (const bf16*)table, scale}, aligned, w, x, T, C, groups,
                             eps, stream);
  return NIB_ERR_BAD_ARGUMENT;
}
