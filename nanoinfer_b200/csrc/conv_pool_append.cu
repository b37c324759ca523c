// What lies between the projection and the scores of an attention whose keys pass a short convolution, are normed per
// head, double as the values, and are kept once more as means over blocks of positions:
//   u      = the projected queries and keys (32-bit columns, all query heads, then all key heads)
//   y_t,c  = sum_j w[j, c] u_(t - taps + 1 + j), c          (what lies before the entry's first row: the request's state)
//   q, k   = y over its root mean square per head (eps inside the root, no weight; optional)
//   cache  : k to plane 0 and the key head's y itself to plane 1 of the row's slot; rows of hd values, zeros behind dim
//   pooled : with pool > 0, the row that ends a block of `pool` positions also writes the block's mean key and mean value,
//            means of what the cache holds, as row (position / pool) of the request's pooled pages (same cache)
// in one kernel, and in a step whose entries are one row each the convolution's state as well.
//
// A block owns a row and eight heads, a warp a head; the pooled rows are made by blocks of their own (a row and a key head,
// which leave at once where the row ends no block) unless every entry is one row, where the block that owns the key head does
// it.  The keys of a pooled block that came with this step may not be in the cache yet (other blocks of the launch write them):
// they are made again from the projection, with the same rounding; those of earlier steps are read from the cache.  The eight
// warps share a block's positions (by index modulo eight) and add up in warp order, so a mean does not depend on how the
// prompt was cut.  The usual numbers of taps are compiled in, so that all of a head's loads travel together.
#include "api.h"
#include "common.cuh"

namespace nib {

constexpr int CP_WARPS = 8;

template <typename T>
struct ConvPoolParams {
  const float* proj;
  int ld, taps;
  const float* w;              // [taps][channels]
  float* state;                // a request's row: the last taps - 1 projected rows, oldest first
  long long state_stride;
  const int* entry_start;
  const int* entry_slot;
  const int* positions;
  const int* row_entry;
  int n_head, n_kv_head, dim, hd, norm;
  float eps;
  T* q_out;
  int ldq;
  T* cache;
  const int* block_table;
  const int* pool_table;
  int max_blocks, page_size, n_pages, pool, shift_state;
  int head_blocks;             // blocks of eight heads a row; behind them, a block a key head for the pooled rows
  int* status;
};

template <typename T, int ND, int TAPS>
__global__ void __launch_bounds__(CP_WARPS * 32)
conv_pool_append_kernel(const ConvPoolParams<T> prm) {
  pdl_trigger();
  extern __shared__ float means[];                 // [warps][key | value][hd]
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int entry = prm.row_entry[t];
  if (entry < 0) return;                           // a row of no request
  const int pos = prm.positions[t], i = t - prm.entry_start[entry];
  const int dim = prm.dim, hd = prm.hd, taps = TAPS > 0 ? TAPS : prm.taps, H = prm.n_head, G = prm.n_kv_head;
  const bool pools = (int)blockIdx.y >= prm.head_blocks, ends = prm.pool > 0 && (pos + 1) % prm.pool == 0;
  if (pools && !ends) return;
  const int channels = (H + G) * dim;
  float* st = prm.state + (size_t)prm.entry_slot[entry] * prm.state_stride;
  const int* table = prm.block_table + (size_t)entry * prm.max_blocks;
  auto slot_of = [&](const int* tab, int row) -> T* {   // key head 0's key of a row; null where there is no page
    const int page = tab[row / prm.page_size];
    if (page < 0 || page >= prm.n_pages) {
      *prm.status = NIB_STATUS_BAD_PAGE;
      return nullptr;
    }
    return prm.cache + kv_offset(page, 0, 0, row % prm.page_size, G, prm.page_size, hd);
  };
  const size_t head_stride = (size_t)prm.page_size * hd, plane = (size_t)G * head_stride;
  pdl_wait();

  // the convolution's output of head `unit` for the row `back` rows above t (which is one of this entry's), in v; returns
  // what makes it a normed head
  auto head_row = [&](int unit, int back, float* v) -> float {
    float q = 0.0f;
#pragma unroll
    for (int n = 0; n < ND; ++n) {
      const int d = lane + 32 * n, c = unit * dim + d;
      float acc = 0.0f;
      if (d < dim) {
        auto at = [&](int j) -> const float* {
          const int src = i - back - (taps - 1 - j);
          return src >= 0 ? prm.proj + (size_t)(t - back - (taps - 1 - j)) * prm.ld + c : st + (size_t)(taps - 1 + src) * channels + c;
        };
        if constexpr (TAPS > 0) {
          float x[TAPS], w[TAPS];
#pragma unroll
          for (int j = 0; j < TAPS; ++j) {
            x[j] = *at(j);
            w[j] = prm.w[(size_t)j * channels + c];
          }
#pragma unroll
          for (int j = 0; j < TAPS; ++j) acc = fmaf(w[j], x[j], acc);
        } else {
          for (int j = 0; j < taps; ++j) acc = fmaf(prm.w[(size_t)j * channels + c], *at(j), acc);
        }
      }
      v[n] = acc;
      q += acc * acc;
    }
    return prm.norm ? 1.0f / sqrtf(warp_sum(q) / (float)dim + prm.eps) : 1.0f;
  };

  const int u0 = blockIdx.y * CP_WARPS, unit = u0 + warp;
  if (!pools && unit < H + G) {
    float v[ND];
    const float r = head_row(unit, 0, v);
    if (unit < H) {
      T* dst = prm.q_out + (size_t)t * prm.ldq + (size_t)unit * hd;
#pragma unroll
      for (int n = 0; n < ND; ++n)
        if (lane + 32 * n < hd) dst[lane + 32 * n] = from_float<T>(v[n] * r);
    } else {
      T* dst = slot_of(table, pos);
      if (dst != nullptr) {
        dst += (unit - H) * head_stride;
#pragma unroll
        for (int n = 0; n < ND; ++n)
          if (lane + 32 * n < hd) {
            dst[lane + 32 * n] = from_float<T>(v[n] * r);
            dst[plane + lane + 32 * n] = from_float<T>(v[n]);
          }
      }
    }
  }
  if (ends && (pools || prm.shift_state)) {
    const int P = prm.pool, first = pos + 1 - P;
    const int g0 = pools ? (int)blockIdx.y - prm.head_blocks : max(u0 - H, 0);
    const int g1 = pools ? g0 + 1 : min(u0 + CP_WARPS - H, G);
    for (int g = g0; g < g1; ++g) {
      float ks[ND], vs[ND];
#pragma unroll
      for (int n = 0; n < ND; ++n) ks[n] = vs[n] = 0.0f;
      for (int p = first + warp; p <= pos; p += CP_WARPS) {
        if (pos - p <= i) {                        // came with this step
          float v[ND];
          const float r = head_row(H + g, pos - p, v);
#pragma unroll
          for (int n = 0; n < ND; ++n) {
            ks[n] += to_float(from_float<T>(__fmul_rn(v[n], r)));   // (the cached value: no multiply-add across it)
            vs[n] += to_float(from_float<T>(v[n]));
          }
        } else {
          const T* src = slot_of(table, p);
          if (src == nullptr) continue;
          src += g * head_stride;
#pragma unroll
          for (int n = 0; n < ND; ++n)
            if (lane + 32 * n < dim) {
              ks[n] += to_float(src[lane + 32 * n]);
              vs[n] += to_float(src[plane + lane + 32 * n]);
            }
        }
      }
      __syncthreads();                             // (the head before is done with the means)
#pragma unroll
      for (int n = 0; n < ND; ++n)
        if (lane + 32 * n < hd) {
          means[(warp * 2) * hd + lane + 32 * n] = ks[n];
          means[(warp * 2 + 1) * hd + lane + 32 * n] = vs[n];
        }
      __syncthreads();
      T* dst = slot_of(prm.pool_table + (size_t)entry * prm.max_blocks, pos / P);
      if (dst != nullptr)
        for (int x = threadIdx.x; x < 2 * hd; x += CP_WARPS * 32) {
          float s = 0.0f;
#pragma unroll
          for (int w = 0; w < CP_WARPS; ++w) s += means[w * 2 * hd + x];
          dst[g * head_stride + (x < hd ? x : plane + x - hd)] = from_float<T>(s / (float)P);
        }
    }
  }
  if (prm.shift_state && taps > 1) {               // the entry's only row: the state moves on by one, once all have read it
    __syncthreads();
    const int c1 = min(u0 + CP_WARPS, H + G) * dim;
    for (int c = u0 * dim + threadIdx.x; c < c1; c += CP_WARPS * 32) {
      for (int s = 0; s + 2 < taps; ++s) st[(size_t)s * channels + c] = st[(size_t)(s + 1) * channels + c];
      st[(size_t)(taps - 2) * channels + c] = prm.proj[(size_t)t * prm.ld + c];
    }
  }
}

template <typename T, int TAPS>
static int launch_conv_pool_append(const ConvPoolParams<T>& prm, int n_rows, cudaStream_t stream) {
  const dim3 grid(n_rows, prm.head_blocks + (prm.pool > 0 && !prm.shift_state ? prm.n_kv_head : 0)), block(CP_WARPS * 32);
  const size_t smem = prm.pool > 0 ? (size_t)CP_WARPS * 2 * prm.hd * sizeof(float) : 0;
  if (prm.hd <= 64) launch_pdl(conv_pool_append_kernel<T, 2, TAPS>, grid, block, smem, stream, prm);
  else if (prm.hd <= 128) launch_pdl(conv_pool_append_kernel<T, 4, TAPS>, grid, block, smem, stream, prm);
  else launch_pdl(conv_pool_append_kernel<T, 8, TAPS>, grid, block, smem, stream, prm);
  NIB_LAUNCH_CHECK();
}
template <typename T>
static int pick_conv_pool_append(const ConvPoolParams<T>& prm, int n_rows, cudaStream_t stream) {
  switch (prm.taps) {
    case 1: return launch_conv_pool_append<T, 1>(prm, n_rows, stream);
    case 2: return launch_conv_pool_append<T, 2>(prm, n_rows, stream);
    case 3: return launch_conv_pool_append<T, 3>(prm, n_rows, stream);
    case 4: return launch_conv_pool_append<T, 4>(prm, n_rows, stream);
  }
  return launch_conv_pool_append<T, 0>(prm, n_rows, stream);
}

}  // namespace nib

using namespace nib;

// proj: 32-bit rows whose first (n_head + n_kv_head) * dim columns are the projected queries and keys; w [taps][channels];
// state may be null with one tap; cache: one layer [n_pages, 2, n_kv_head, page_size, hd], dim <= hd <= 256.  pool_table: the
// pages of the requests' pooled rows, max_blocks apart like block_table's (null with pool 0).  shift_state: every entry of the
// step is one row, and the kernel moves the state on itself (otherwise nib_short_conv_state does it behind).
extern "C" int nib_conv_pool_append(int dtype, const float* proj, int ld, int taps, const float* w, float* state,
                                    long long state_stride, const int* entry_start, const int* entry_slot,
                                    const int* positions, const int* row_entry, int n_head, int n_kv_head, int dim, int hd,
                                    int norm, float eps, void* q_out, int ldq, void* cache, const int* block_table,
                                    const int* pool_table, int max_blocks, int page_size, int n_pages, int pool,
                                    int shift_state, int T, int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (taps < 1 || taps > 64 || dim <= 0 || dim > hd || hd > 256 || n_head + 2 * n_kv_head > 65535)
    return NIB_ERR_UNSUPPORTED_SIZE;
  if (n_head <= 0 || n_kv_head <= 0 || page_size <= 0 || pool < 0 || (pool > 0 && pool_table == nullptr) || cache == nullptr ||
      (taps > 1 && state == nullptr))
    return NIB_ERR_BAD_ARGUMENT;
  auto fill = [&](auto* prm) {
    prm->proj = proj; prm->ld = ld; prm->taps = taps; prm->w = w; prm->state = state; prm->state_stride = state_stride;
    prm->entry_start = entry_start; prm->entry_slot = entry_slot; prm->positions = positions; prm->row_entry = row_entry;
    prm->n_head = n_head; prm->n_kv_head = n_kv_head; prm->dim = dim; prm->hd = hd; prm->norm = norm; prm->eps = eps;
    prm->ldq = ldq; prm->block_table = block_table; prm->pool_table = pool_table; prm->max_blocks = max_blocks;
    prm->page_size = page_size; prm->n_pages = n_pages; prm->pool = pool; prm->shift_state = shift_state;
    prm->status = status;
    prm->head_blocks = (n_head + n_kv_head + CP_WARPS - 1) / CP_WARPS;
  };
  if (dtype == DT_F32) {
    ConvPoolParams<float> prm;
    fill(&prm);
    prm.q_out = (float*)q_out; prm.cache = (float*)cache;
    return pick_conv_pool_append(prm, T, stream);
  }
  if (dtype == DT_BF16) {
    ConvPoolParams<bf16> prm;
    fill(&prm);
    prm.q_out = (bf16*)q_out; prm.cache = (bf16*)cache;
    return pick_conv_pool_append(prm, T, stream);
  }
  return NIB_ERR_BAD_ARGUMENT;
}
