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
// A block owns a few rows and eight heads, a warp a head; the pooled rows are made by blocks of their own (a block of positions
// and a key head, found from the entries' first positions) unless every entry is one row, where the block that owns the key
// head does it.  The keys of a pooled block that came with this step may not be in the cache yet (other blocks of the launch
// write them): they are made again from the projection, with the same rounding; those of earlier steps are read from the cache.
// The eight warps share a block's positions (by index modulo eight) and add up in warp order, so a mean does not depend on how
// the prompt was cut.  The usual numbers of taps are compiled in, so that all of a head's loads travel together.
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
  const int* entry_pos0;
  const int* entry_slot;
  int n_rows, n_entries;
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
  int head_blocks;             // blocks of eight heads a group of rows
  int row_blocks;              // groups of rows; the blocks behind all of these make the pooled rows
  int* status;
};

// ND: values of a head a lane owns (hd <= 32 ND); R: rows of a block
template <typename T, int ND, int TAPS, int R>
__global__ void __launch_bounds__(CP_WARPS * 32)
conv_pool_append_kernel(const ConvPoolParams<T> prm) {
  pdl_trigger();
  extern __shared__ float means[];                 // [warps][key | value][hd]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int dim = prm.dim, hd = prm.hd, taps = TAPS > 0 ? TAPS : prm.taps, H = prm.n_head, G = prm.n_kv_head;
  const int channels = (H + G) * dim, P = prm.pool;
  const size_t head_stride = (size_t)prm.page_size * hd, plane = (size_t)G * head_stride;
  auto slot_of = [&](const int* tab, int entry, int row) -> T* {   // key head 0's key of a row; null where there is no page
    const int page = tab[(size_t)entry * prm.max_blocks + row / prm.page_size];
    if (page < 0 || page >= prm.n_pages) {
      *prm.status = NIB_STATUS_BAD_PAGE;
      return nullptr;
    }
    return prm.cache + kv_offset(page, 0, 0, row % prm.page_size, G, prm.page_size, hd);
  };
  // the convolution's output of head `unit` for row t, the i-th of its entry (whose state is st), in v; returns this lane's
  // part of its sum of squares
  auto conv_row = [&](int unit, int t, int i, const float* st, float* v) -> float {
    float q = 0.0f;
#pragma unroll
    for (int n = 0; n < ND; ++n) {
      const int d = lane + 32 * n, c = unit * dim + d;
      float acc = 0.0f;
      if (d < dim) {
        auto at = [&](int j) -> const float* {
          const int src = i - (taps - 1 - j);
          return src >= 0 ? prm.proj + (size_t)(t - (taps - 1 - j)) * prm.ld + c : st + (size_t)(taps - 1 + src) * channels + c;
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
    return q;
  };
  auto inv_rms = [&](float q) -> float { return prm.norm ? 1.0f / sqrtf(warp_sum(q) / (float)dim + prm.eps) : 1.0f; };
  // the mean key and value of the block of positions that ends at `pos`, row t, the i-th of its entry; for key head g
  auto pool_block = [&](int entry, int t, int i, int pos, const float* st, int g) {
    float ks[ND], vs[ND];
#pragma unroll
    for (int n = 0; n < ND; ++n) ks[n] = vs[n] = 0.0f;
    for (int p = pos + 1 - P + warp; p <= pos; p += CP_WARPS) {
      const int back = pos - p;
      if (back <= i) {                             // came with this step
        float v[ND];
        const float r = inv_rms(conv_row(H + g, t - back, i - back, st, v));
#pragma unroll
        for (int n = 0; n < ND; ++n) {
          ks[n] += to_float(from_float<T>(__fmul_rn(v[n], r)));   // (the cached value: no multiply-add across it)
          vs[n] += to_float(from_float<T>(v[n]));
        }
      } else {
        const T* src = slot_of(prm.block_table, entry, p);
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
    __syncthreads();                               // (the head before is done with the means)
#pragma unroll
    for (int n = 0; n < ND; ++n)
      if (lane + 32 * n < hd) {
        means[(warp * 2) * hd + lane + 32 * n] = ks[n];
        means[(warp * 2 + 1) * hd + lane + 32 * n] = vs[n];
      }
    __syncthreads();
    T* dst = slot_of(prm.pool_table, entry, pos / P);
    if (dst != nullptr)
      for (int x = threadIdx.x; x < 2 * hd; x += CP_WARPS * 32) {
        float s = 0.0f;
#pragma unroll
        for (int w = 0; w < CP_WARPS; ++w) s += means[w * 2 * hd + x];
        dst[g * head_stride + (x < hd ? x : plane + x - hd)] = from_float<T>(s / (float)P);
      }
  };

  const int n_head_blocks = prm.row_blocks * prm.head_blocks;
  if ((int)blockIdx.x >= n_head_blocks) {
    // ---- a pooled row: the b-th block of positions that ends in this step, entry by entry
    int b = ((int)blockIdx.x - n_head_blocks) / G;
    const int g = ((int)blockIdx.x - n_head_blocks) % G;
    int e = 0, first = 0, t0 = 0;
    for (; e < prm.n_entries; ++e) {
      t0 = prm.entry_start[e];
      first = prm.entry_pos0[e];
      const int ends = (first + prm.entry_start[e + 1] - t0) / P - first / P;
      if (b < ends) break;
      b -= ends;
    }
    if (e >= prm.n_entries) return;                // (the launch has blocks for the most that can end)
    const int pos = (first / P + b + 1) * P - 1, i = pos - first;
    pdl_wait();
    pool_block(e, t0 + i, i, pos, prm.state + (size_t)prm.entry_slot[e] * prm.state_stride, g);
    return;
  }
  const int row0 = (int)blockIdx.x / prm.head_blocks * R, u0 = (int)blockIdx.x % prm.head_blocks * CP_WARPS, unit = u0 + warp;
  int entry[R], pos[R], start[R];
  float* st[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    entry[r] = row0 + r < prm.n_rows ? prm.row_entry[row0 + r] : -1;   // (-1: a row of no request, too)
    pos[r] = start[r] = 0;
    st[r] = prm.state;
    if (entry[r] >= 0) {
      pos[r] = prm.positions[row0 + r];
      start[r] = prm.entry_start[entry[r]];
      st[r] = prm.state + (size_t)prm.entry_slot[entry[r]] * prm.state_stride;
    }
  }
  pdl_wait();
  if (unit < H + G) {
    float v[R][ND], q[R];
#pragma unroll
    for (int r = 0; r < R; ++r) q[r] = entry[r] >= 0 ? conv_row(unit, row0 + r, row0 + r - start[r], st[r], v[r]) : 0.0f;
#pragma unroll
    for (int r = 0; r < R; ++r) q[r] = inv_rms(q[r]);
#pragma unroll
    for (int r = 0; r < R; ++r) {
      if (entry[r] < 0) continue;
      if (unit < H) {
        T* dst = prm.q_out + (size_t)(row0 + r) * prm.ldq + (size_t)unit * hd;
#pragma unroll
        for (int n = 0; n < ND; ++n)
          if (lane + 32 * n < hd) dst[lane + 32 * n] = from_float<T>(v[r][n] * q[r]);
      } else {
        T* dst = slot_of(prm.block_table, entry[r], pos[r]);
        if (dst == nullptr) continue;
        dst += (unit - H) * head_stride;
#pragma unroll
        for (int n = 0; n < ND; ++n)
          if (lane + 32 * n < hd) {
            dst[lane + 32 * n] = from_float<T>(v[r][n] * q[r]);
            dst[plane + lane + 32 * n] = from_float<T>(v[r][n]);
          }
      }
    }
  }
  if (!prm.shift_state || entry[0] < 0) return;
  // ---- every entry is one row (R is 1): its pooled row, and its state moves on by one once all have read it
  if (P > 0 && (pos[0] + 1) % P == 0)
    for (int g = max(u0 - H, 0); g < min(u0 + CP_WARPS - H, G); ++g) pool_block(entry[0], row0, row0 - start[0], pos[0], st[0], g);
  if (taps > 1) {
    __syncthreads();
    const int c1 = min(u0 + CP_WARPS, H + G) * dim;
    for (int c = u0 * dim + threadIdx.x; c < c1; c += CP_WARPS * 32) {
      for (int s = 0; s + 2 < taps; ++s) st[0][(size_t)s * channels + c] = st[0][(size_t)(s + 1) * channels + c];
      st[0][(size_t)(taps - 2) * channels + c] = prm.proj[(size_t)row0 * prm.ld + c];
    }
  }
}

template <typename T, int ND, int TAPS, int R>
static void launch_conv_pool_rows(ConvPoolParams<T> prm, cudaStream_t stream) {
  prm.row_blocks = (prm.n_rows + R - 1) / R;
  // at most so many blocks of positions end in the step: one for every `pool` rows, and one more an entry
  const int ends = prm.pool > 0 && !prm.shift_state ? prm.n_rows / prm.pool + prm.n_entries : 0;
  launch_pdl(conv_pool_append_kernel<T, ND, TAPS, R>, dim3(prm.row_blocks * prm.head_blocks + ends * prm.n_kv_head),
             dim3(CP_WARPS * 32), prm.pool > 0 ? (size_t)CP_WARPS * 2 * prm.hd * sizeof(float) : 0, stream, prm);
}
template <typename T, int TAPS>
static int launch_conv_pool_append(const ConvPoolParams<T>& prm, cudaStream_t stream) {
  if (prm.hd <= 64) {
    if (prm.shift_state) launch_conv_pool_rows<T, 2, TAPS, 1>(prm, stream);
    else launch_conv_pool_rows<T, 2, TAPS, 4>(prm, stream);
  } else if (prm.hd <= 128) {
    if (prm.shift_state) launch_conv_pool_rows<T, 4, TAPS, 1>(prm, stream);
    else launch_conv_pool_rows<T, 4, TAPS, 2>(prm, stream);
  } else {
    launch_conv_pool_rows<T, 8, TAPS, 1>(prm, stream);
  }
  NIB_LAUNCH_CHECK();
}
template <typename T>
static int pick_conv_pool_append(const ConvPoolParams<T>& prm, cudaStream_t stream) {
  switch (prm.taps) {
    case 1: return launch_conv_pool_append<T, 1>(prm, stream);
    case 2: return launch_conv_pool_append<T, 2>(prm, stream);
    case 3: return launch_conv_pool_append<T, 3>(prm, stream);
    case 4: return launch_conv_pool_append<T, 4>(prm, stream);
  }
  return launch_conv_pool_append<T, 0>(prm, stream);
}

}  // namespace nib

using namespace nib;

// proj: 32-bit rows whose first (n_head + n_kv_head) * dim columns are the projected queries and keys; w [taps][channels];
// state may be null with one tap; cache: one layer [n_pages, 2, n_kv_head, page_size, hd], dim <= hd <= 256.  pool_table: the
// pages of the requests' pooled rows, max_blocks apart like block_table's (null with pool 0).  shift_state: every entry of the
// step is one row, and the kernel moves the state on itself (otherwise nib_short_conv_state does it behind).
extern "C" int nib_conv_pool_append(int dtype, const float* proj, int ld, int taps, const float* w, float* state,
                                    long long state_stride, const int* entry_start, const int* entry_pos0,
                                    const int* entry_slot, int n_entries,
                                    const int* positions, const int* row_entry, int n_head, int n_kv_head, int dim, int hd,
                                    int norm, float eps, void* q_out, int ldq, void* cache, const int* block_table,
                                    const int* pool_table, int max_blocks, int page_size, int n_pages, int pool,
                                    int shift_state, int T, int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (taps < 1 || taps > 64 || dim <= 0 || dim > hd || hd > 256 || n_entries < 0)
    return NIB_ERR_UNSUPPORTED_SIZE;
  if (n_head <= 0 || n_kv_head <= 0 || page_size <= 0 || pool < 0 || (pool > 0 && pool_table == nullptr) || cache == nullptr ||
      (taps > 1 && state == nullptr))
    return NIB_ERR_BAD_ARGUMENT;
  auto fill = [&](auto* prm) {
    prm->proj = proj; prm->ld = ld; prm->taps = taps; prm->w = w; prm->state = state; prm->state_stride = state_stride;
    prm->entry_start = entry_start; prm->entry_pos0 = entry_pos0;
    prm->entry_slot = entry_slot; prm->n_rows = T; prm->n_entries = n_entries; prm->row_blocks = 0;
    prm->positions = positions; prm->row_entry = row_entry;
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
    return pick_conv_pool_append(prm, stream);
  }
  if (dtype == DT_BF16) {
    ConvPoolParams<bf16> prm;
    fill(&prm);
    prm.q_out = (bf16*)q_out; prm.cache = (bf16*)cache;
    return pick_conv_pool_append(prm, stream);
  }
  return NIB_ERR_BAD_ARGUMENT;
}
