// The minimal gated recurrent unit: a recurrence whose gate and candidate read the current token only, so that every
// channel of the state is a first-order linear recurrence of its own:
//   z = sigmoid(z logit);   c = u + 1/2 where u >= 0, sigmoid(u) where u < 0;   S <- S + z (c - S)
//   out = S silu(g)
// The three logits of a row (biases added) lie at three column offsets of the 32-bit projection; S (one float a channel,
// zero at a sequence's start) comes from and goes to the request's state slot; all arithmetic is 32-bit.
//
// A linear recurrence can be cut in time.  Thirty-two channels of one entry (a lane each) belong to a cluster of up to eight
// blocks of sixteen warps; a chunk of up to 1024 rows is cut into runs of at most eight rows, a warp each, block after block.
// A warp first walks its run from S = 0, keeping the run's gates and candidates in registers, which gives the run's own
// result b and the fraction f of an incoming state that it forgets (f <- f + z (1 - f), kept as the fraction FORGOTTEN: of a
// slow channel's remaining fraction, a number next to 1, a float would lose what is forgotten).  Runs compose:
// S_out = b + S_in - f S_in.  A block chains its warps' runs through shared memory, the cluster its blocks' through
// distributed shared memory, and every warp then walks its run once more, in registers, from its true incoming state and
// writes its rows.  A step of single tokens takes a form of its own with nothing to chain.
#include "api.h"
#include "common.cuh"

namespace nib {

__device__ __forceinline__ float mg_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }

constexpr int MG_WARPS = 16, MG_ROWS = 8, MG_MAX_CLUSTER = 8;

template <typename OutT>
__global__ void __launch_bounds__(MG_WARPS * 32)
min_gru_kernel(const float* proj, int ld, int z_off, int u_off, int g_off, int width, float* state,
               long long state_stride, const int* __restrict__ entry_start, const int* __restrict__ entry_slot, OutT* out,
               int ldo, int cluster) {
  pdl_trigger();
  __shared__ float run_b[MG_WARPS][32], run_f[MG_WARPS][32];
  __shared__ float blk[2][2][32];                   // [chunk parity][b, f][channel] of the whole block's runs
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int rank = cluster > 1 ? blockIdx.x % cluster : 0;
  const int e = blockIdx.y, c = blockIdx.x / cluster * 32 + lane;
  const bool live = c < width;
  const int r_begin = entry_start[e], r_end = entry_start[e + 1];
  pdl_wait();
  float* slot = state + (size_t)entry_slot[e] * state_stride;
  float carry = live ? slot[c] : 0.0f;              // the state ahead of the chunk, the same in every warp of the cluster
  const int n_runs = cluster * MG_WARPS;
  int parity = 0;
  for (int r0 = r_begin; r0 < r_end; r0 += n_runs * MG_ROWS, parity ^= 1) {
    // consecutive rows to consecutive runs, and no run without rows while another has two more
    const int n = min(n_runs * MG_ROWS, r_end - r0);
    const int per = (n + n_runs - 1) / n_runs;
    const int a = r0 + (rank * MG_WARPS + warp) * per, rows = max(0, min(per, r0 + n - a));
    float z[MG_ROWS], cand[MG_ROWS], g[MG_ROWS];
#pragma unroll
    for (int i = 0; i < MG_ROWS; ++i) {
      if (i < rows && live) {
        const float* p = proj + (size_t)(a + i) * ld + c;
        z[i] = p[z_off];
        cand[i] = p[u_off];
        g[i] = p[g_off];
      }
    }
    float b = 0.0f, f = 0.0f;
#pragma unroll
    for (int i = 0; i < MG_ROWS; ++i) {
      if (i < rows && live) {
        z[i] = mg_sigmoid(z[i]);
        cand[i] = cand[i] >= 0.0f ? cand[i] + 0.5f : mg_sigmoid(cand[i]);
        b = fmaf(z[i], cand[i] - b, b);
        f = fmaf(z[i], 1.0f - f, f);
      }
    }
    __syncthreads();                                // the chunk before is done with the runs' results
    run_b[warp][lane] = b;
    run_f[warp][lane] = f;
    __syncthreads();
    // the block's runs chained: what lies ahead of this warp's run, and the whole block
    float B = 0.0f, F = 0.0f, Bw = 0.0f, Fw = 0.0f;
#pragma unroll
    for (int w = 0; w < MG_WARPS; ++w) {
      if (w == warp) {
        Bw = B;
        Fw = F;
      }
      const float rf = run_f[w][lane];
      B = run_b[w][lane] + fmaf(-rf, B, B);
      F = fmaf(rf, 1.0f - F, F);
    }
    float S = carry;                                // the state ahead of this block
    if (cluster == 1) {
      carry = B + fmaf(-F, carry, carry);
    } else {
      if (warp == 0) {
        blk[parity][0][lane] = B;
        blk[parity][1][lane] = F;
      }
      cluster_arrive();
      cluster_wait();
      for (int k = 0; k < cluster; ++k) {
        if (k == rank) S = carry;
        const float kb = __uint_as_float(cluster_load(cluster_addr(&blk[parity][0][lane], k)));
        const float kf = __uint_as_float(cluster_load(cluster_addr(&blk[parity][1][lane], k)));
        carry = kb + fmaf(-kf, carry, carry);
      }
    }
    S = Bw + fmaf(-Fw, S, S);                       // ... and ahead of this warp's run
#pragma unroll
    for (int i = 0; i < MG_ROWS; ++i) {
      if (i < rows && live) {
        S = fmaf(z[i], cand[i] - S, S);
        out[(size_t)(a + i) * ldo + c] = from_float<OutT>(S * (g[i] * mg_sigmoid(g[i])));
      }
    }
  }
  if (cluster > 1) {                                // nobody leaves while its shared memory is read
    __syncthreads();
    cluster_arrive();
    cluster_wait();
  }
  if (rank == 0 && warp == 0 && live) slot[c] = carry;
}

// Single tokens: entry e is row e; a thread a (row, channel).
template <typename OutT>
__global__ void __launch_bounds__(128)
min_gru_token_kernel(const float* proj, int ld, int z_off, int u_off, int g_off, int width, float* state,
                     long long state_stride, const int* __restrict__ entry_slot, OutT* out, int ldo) {
  pdl_trigger();
  const int t = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int s = entry_slot[t];
  pdl_wait();
  if (c >= width) return;
  const float* p = proj + (size_t)t * ld + c;
  float* slot = state + (size_t)s * state_stride + c;
  const float z = mg_sigmoid(p[z_off]), u = p[u_off], g = p[g_off], old = *slot;
  const float cand = u >= 0.0f ? u + 0.5f : mg_sigmoid(u);
  const float S = fmaf(z, cand - old, old);
  *slot = S;
  out[(size_t)t * ldo + c] = from_float<OutT>(S * (g * mg_sigmoid(g)));
}

template <typename OutT>
static int launch_min_gru(const float* proj, int ld, int z_off, int u_off, int g_off, int width, float* state,
                          long long state_stride, const int* entry_start, const int* entry_slot, int n_entries, int n_rows,
                          OutT* out, int ldo, cudaStream_t stream) {
  if (n_rows == n_entries)     // every entry has one row
    launch_pdl(min_gru_token_kernel<OutT>, dim3((width + 127) / 128, n_entries), dim3(128), 0, stream, proj, ld, z_off, u_off,
               g_off, width, state, state_stride, entry_slot, out, ldo);
  else
  {
    // blocks of a cluster: as many as the step's rows can fill (a function of the step's shape alone)
    int cluster = 1;
    while (cluster < MG_MAX_CLUSTER && n_rows > cluster * MG_WARPS * MG_ROWS) cluster *= 2;
    launch_pdl_cluster(min_gru_kernel<OutT>, dim3((width + 31) / 32 * cluster, n_entries), dim3(MG_WARPS * 32), 0, stream,
                       cluster, proj, ld, z_off, u_off, g_off, width, state, state_stride, entry_start, entry_slot, out, ldo,
                       cluster);
  }
  NIB_LAUNCH_CHECK();
}

}  // namespace nib

using namespace nib;

// n_rows: the rows of the step (at least one an entry; rows of no request may follow the entries').
extern "C" int nib_min_gru(int out_dtype, const float* proj, int ld, int z_off, int u_off, int g_off, int width,
                           float* state, long long state_stride, const int* entry_start, const int* entry_slot,
                           int n_entries, int n_rows, void* out, int ldo, cudaStream_t stream) {
  if (n_entries <= 0) return 0;
  if (width <= 0 || n_rows < n_entries) return NIB_ERR_BAD_ARGUMENT;
  if (n_entries > 65535) return NIB_ERR_UNSUPPORTED_SIZE;
  if (out_dtype == DT_F32)
    return launch_min_gru<float>(proj, ld, z_off, u_off, g_off, width, state, state_stride, entry_start, entry_slot,
                                 n_entries, n_rows, (float*)out, ldo, stream);
  if (out_dtype == DT_BF16)
    return launch_min_gru<bf16>(proj, ld, z_off, u_off, g_off, width, state, state_stride, entry_start, entry_slot,
                                n_entries, n_rows, (bf16*)out, ldo, stream);
  return NIB_ERR_BAD_ARGUMENT;
}
