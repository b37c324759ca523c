// What follows the two attention maps of a differential head: the second map's output times one number is subtracted
// from the first's, the difference is divided by its root mean square over the head's values (eps inside the root, no
// weight) and multiplied by a constant:
//   o = a[t, 2h] - lambda a[t, 2h + 1];   out[t, h] = mul o / sqrt(mean(o^2) + eps)
// The maps' outputs are 32-bit heads of hd values of which the first vdim count (the attention kernels leave them so
// with AttnExtras::out32: the difference of two nearly equal results is taken before anything is rounded).  A warp a
// (row, head).  Single decoded tokens in bfloat16 have it done where their pieces of keys are merged
// (attention_group_mma.cu).
#include "api.h"
#include "common.cuh"

namespace nib {

constexpr int DC_MAX = 8;   // values a lane holds: vdim <= 256

template <typename OutT>
__global__ void __launch_bounds__(256)
diff_combine_kernel(const float* a, int lda, const int* __restrict__ rows, int n_head, int hd, int vdim, float lambda,
                    float eps, float mul, OutT* out, int ldo, int T) {
  pdl_trigger();
  const int lane = threadIdx.x & 31;
  const int unit = blockIdx.x * 8 + (threadIdx.x >> 5);
  const int r = unit / n_head, h = unit % n_head;
  const int t = r < T && rows ? rows[r] : r;
  pdl_wait();
  if (r >= T) return;
  const float* a1 = a + (size_t)t * lda + (size_t)(2 * h) * hd;
  const float* a2 = a1 + hd;
  float o[DC_MAX], q = 0.0f;
#pragma unroll
  for (int i = 0; i < DC_MAX; ++i) {
    const int d = lane + 32 * i;
    o[i] = d < vdim ? fmaf(-lambda, a2[d], a1[d]) : 0.0f;
    q += o[i] * o[i];
  }
  const float f = mul / sqrtf(warp_sum(q) / (float)vdim + eps);
  OutT* dst = out + (size_t)t * ldo + (size_t)h * vdim;
#pragma unroll
  for (int i = 0; i < DC_MAX; ++i) {
    const int d = lane + 32 * i;
    if (d < vdim) dst[d] = from_float<OutT>(o[i] * f);
  }
}

}  // namespace nib

using namespace nib;

// rows: the T rows to process (nullptr: rows 0..T-1).
extern "C" int nib_diff_combine(int out_dtype, const float* a, int lda, const int* rows, int n_head, int hd, int vdim, float lambda,
                                float eps, float mul, void* out, int ldo, int T, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (n_head <= 0 || vdim <= 0 || vdim > hd) return NIB_ERR_BAD_ARGUMENT;
  if (vdim > 32 * DC_MAX) return NIB_ERR_UNSUPPORTED_SIZE;
  const dim3 grid((unsigned)(((long long)T * n_head + 7) / 8));
  if (out_dtype == DT_F32)
    launch_pdl(diff_combine_kernel<float>, grid, dim3(256), 0, stream, a, lda, rows, n_head, hd, vdim, lambda, eps, mul,
               (float*)out, ldo, T);
  else if (out_dtype == DT_BF16)
    launch_pdl(diff_combine_kernel<bf16>, grid, dim3(256), 0, stream, a, lda, rows, n_head, hd, vdim, lambda, eps, mul,
               (bf16*)out, ldo, T);
  else
    return NIB_ERR_BAD_ARGUMENT;
  NIB_LAUNCH_CHECK();
}
