// One step of single tokens of a time-mixing recurrence (csrc/gla.cu names the equations) as ONE kernel: what stands
// between the products r, k, v, g, w1 of a step in which every request brings one token and the output product.
// The products leave float32 split sums [splits][groups x group_rows][N], N = H D: group 0 r, 1 k, 2 v, 3 g, 4 the
// low-rank input of the decay (its first ``rank`` columns); token t is row t of each group.  One block a (request, head):
//
//   r, k, v, g, l <- the sums of the splits;     a = exp(-exp(W2 tanh(l) + w0));
//   o = (S + diag(u) k v^T)^T r;     S <- diag(a) S + k v^T;
//   out = o / rms(o) * weight * silu(g)           in bfloat16.
//
// Everything is float32.  The state and the decay's weights are asked for before the wait on the preceding kernel: the
// weights are constant, and a state is written by a kernel of an EARLIER step only, which is complete (a step starts with
// a copy or with a kernel that nothing overtakes).
// Threads: 16 rows of D / 4 threads; thread (y, q) holds columns 4 q .. 4 q + 3 of the state's rows y, y + 16, ...
#include <math.h>

#include "common.cuh"

namespace {

using namespace tl;

constexpr int ROWS = 16;
constexpr int MAX_D = 128, MAX_RANK = 256, AHEAD = 16;

// the sum of ``splits`` planes, eight loads in flight
__device__ __forceinline__ float sum_splits(const float* p, int splits, size_t plane) {
  float total = 0.f;
  for (int s0 = 0; s0 < splits; s0 += 8) {
    float v[8];
#pragma unroll
    for (int s = 0; s < 8; ++s) v[s] = s0 + s < splits ? p[(size_t)(s0 + s) * plane] : 0.f;
#pragma unroll
    for (int s = 0; s < 8; ++s) total += v[s];
  }
  return total;
}

template <int PER>  // state rows a thread holds: D <= 16 PER
__global__ void __launch_bounds__(ROWS * PER * 4)
time_mixing_step_kernel(const float* __restrict__ sums, int splits, int group_rows, const float* __restrict__ w2t,
                        const float* __restrict__ w0, const float* __restrict__ bonus, const float* __restrict__ weight,
                        const int* __restrict__ slots, float* __restrict__ state, __nv_bfloat16* __restrict__ out,
                        int heads, int dim, int rank, int max_slots, float eps) {
  tl::pdl_launch_dependents();
  constexpr int NT = ROWS * PER * 4;
  __shared__ float s_in[4][MAX_D];  // r, k, v, g
  __shared__ float s_low[MAX_RANK], s_decay[MAX_D], s_o[ROWS][MAX_D], s_sq[MAX_D];
  const int req = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int quads = dim >> 2, N = heads * dim;
  const int y = tid / quads, q = tid - y * quads;
  const bool holds = y < ROWS;
  const int slot = slots[req];
  const bool live = TL_DEBUG_OK(slot >= -1 && slot < max_slots, TL_DEBUG_SLOT, slot) && slot >= 0;
  float* mine = state + ((size_t)(live ? slot : 0) * heads + h) * dim * dim;
  float4 S[PER];
#pragma unroll
  for (int n = 0; n < PER; ++n) {
    const int i = y + n * ROWS;
    S[n] = (live && holds && i < dim) ? *reinterpret_cast<const float4*>(mine + (size_t)i * dim + 4 * q) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  // the decay's second product: ``slices`` threads share a channel's sum over the rank
  const int slices = NT / dim, slice = tid / dim, channel = tid - slice * dim;
  const bool decays = slice < slices;
  float w2[AHEAD];
#pragma unroll
  for (int j = 0; j < AHEAD; ++j) {
    const int at = slice + j * slices;
    w2[j] = (decays && at < rank) ? w2t[(size_t)at * N + h * dim + channel] : 0.f;
  }
  tl::pdl_wait();
  const size_t plane = (size_t)5 * group_rows * N;
  for (int e = tid; e < 4 * dim + rank; e += NT) {
    const int what = e < 4 * dim ? e / dim : 4, c = e - what * dim;
    const float v = sum_splits(sums + ((size_t)what * group_rows + req) * N + (what < 4 ? h * dim + c : c), splits, plane);
    if (what < 4) s_in[what][c] = v;
    else s_low[c] = tanhf(v);
  }
  __syncthreads();
  {
    float z = 0.f;
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {
      const int at = slice + j * slices;
      if (decays && at < rank) z = fmaf(w2[j], s_low[at], z);
    }
    for (int at = slice + AHEAD * slices; decays && at < rank; at += slices)
      z = fmaf(w2t[(size_t)at * N + h * dim + channel], s_low[at], z);
    // slices <= NT / dim; their sums meet in s_o's memory, [slice][channel]
    float* meet = &s_o[0][0];
    if (decays && slice < ROWS) meet[slice * MAX_D + channel] = z;
    __syncthreads();
    if (tid < dim) {
      float total = w0[h * dim + tid];
      for (int s = 0; s < slices && s < ROWS; ++s) total += meet[s * MAX_D + tid];
      s_decay[tid] = expf(-expf(total));
    }
    __syncthreads();
  }
  if (holds) {
    const float4 v = *reinterpret_cast<const float4*>(&s_in[2][4 * q]);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int n = 0; n < PER; ++n) {
      const int i = y + n * ROWS;
      if (i < dim) {
        const float r = s_in[0][i], k = s_in[1][i], a = s_decay[i], u = bonus[h * dim + i];
        const float4 kv = make_float4(k * v.x, k * v.y, k * v.z, k * v.w);
        o.x = fmaf(r, fmaf(u, kv.x, S[n].x), o.x);
        o.y = fmaf(r, fmaf(u, kv.y, S[n].y), o.y);
        o.z = fmaf(r, fmaf(u, kv.z, S[n].z), o.z);
        o.w = fmaf(r, fmaf(u, kv.w, S[n].w), o.w);
        S[n] = make_float4(fmaf(a, S[n].x, kv.x), fmaf(a, S[n].y, kv.y), fmaf(a, S[n].z, kv.z), fmaf(a, S[n].w, kv.w));
        if (live) *reinterpret_cast<float4*>(mine + (size_t)i * dim + 4 * q) = S[n];
      }
    }
    *reinterpret_cast<float4*>(&s_o[y][4 * q]) = o;
  }
  __syncthreads();
  float o = 0.f;
  if (tid < dim) {
    const int rows = dim < ROWS ? dim : ROWS;
    for (int i = 0; i < rows; ++i) o += s_o[i][tid];
    s_sq[tid] = o * o;
  }
  __syncthreads();
  if (tid < dim) {
    float ss = 0.f;
    for (int i = 0; i < dim; i += 4) {  // every thread takes the sum itself (broadcast reads)
      const float4 x = *reinterpret_cast<const float4*>(&s_sq[i]);
      ss += (x.x + x.y) + (x.z + x.w);
    }
    const float g = s_in[3][tid];
    const float value = o / sqrtf(ss / (float)dim + eps) * weight[h * dim + tid] * (g / (1.f + expf(-g)));
    out[(size_t)req * N + h * dim + tid] = __float2bfloat16_rn(live ? value : 0.f);
  }
}

}  // namespace

TL_DEBUG_READER(tl_time_mixing_debug_error)

extern "C" {

int tl_time_mixing_step_supported(int heads, int dim, int rank) {
  return dim % 4 == 0 && dim >= 16 && dim <= MAX_D && rank <= MAX_RANK && rank <= heads * dim && heads <= 65535 ? 1 : 0;
}

// sums: float32 [splits][5 * group_rows][heads * dim]; w2t [rank][heads * dim]; state [max_slots][heads][dim][dim];
// out bfloat16 [requests][heads * dim].
int tl_time_mixing_step(const float* sums, int splits, int group_rows, const float* w2t, const float* w0, const float* bonus,
                        const float* weight, const int* slots, float* state, void* out, int requests, int heads, int dim,
                        int rank, int max_slots, float eps, cudaStream_t stream) {
  if (requests <= 0) return 0;
  if (!tl_time_mixing_step_supported(heads, dim, rank) || splits < 1 || requests > group_rows) return TL_ERR_UNSUPPORTED;
  const dim3 grid(requests, heads);
#define TL_STEP(PER)                                                                                                \
  tl::launch_kernel(time_mixing_step_kernel<PER>, grid, ROWS * PER * 4, 0, stream, sums, splits, group_rows, w2t, w0, bonus, \
                    weight, slots, state, (__nv_bfloat16*)out, heads, dim, rank, max_slots, eps)
  if (dim <= 16) TL_STEP(1);
  else if (dim <= 32) TL_STEP(2);
  else if (dim <= 64) TL_STEP(4);
  else TL_STEP(8);
#undef TL_STEP
  return TL_LAUNCH_CHECK();
}

}  // extern "C"
