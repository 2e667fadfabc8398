// The start of a model's residual streams: a token's embedding row, plus a row of a table of token PAIRS, normed, and
// copied to every stream, in one pass.  One block per token, float32:
//
//   x = table[id] * scale + pairs[row],   row = (previous * mul_prev + id * mul_cur) mod buckets, or ``buckets`` (the last
//                                         row) for the first token of a sequence
//   y = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w (+ b)      (``centre``; without it an RMS norm; w null: y = x)
//   out[t, s] = y for every stream s
//
// The previous token is the one before it in the step, or, for a request's first token of the step, the last token of
// the request's earlier steps, which its slot keeps (``last``, int32 [slots]).  The block that reads the slot is the one
// that then writes the request's last token of this step to it, so no other block races with it.
#include <math.h>

#include "common.cuh"

namespace {

using namespace tl;

constexpr int NT = 256;

template <typename T>
__global__ void __launch_bounds__(NT)
token_embed_kernel(const T* __restrict__ table, const T* __restrict__ pairs, const int* __restrict__ ids,
                   const int* __restrict__ positions, const int* __restrict__ token_req, const int* __restrict__ req_indptr,
                   const int* __restrict__ slots, int* __restrict__ last, int max_slots, int buckets, long long mul_prev,
                   long long mul_cur, const float* __restrict__ weight, const float* __restrict__ bias, float eps, int centre,
                   float* __restrict__ out, int streams, int width, int vocab, float scale) {
  tl::pdl_launch_dependents();
  tl::pdl_wait();
  extern __shared__ __align__(16) float x[];  // width
  __shared__ float scratch[32];
  __shared__ long long pair_row;
  const int t = blockIdx.x;
  const int id = ids[t];
  const bool ok = id >= 0 && id < vocab;
  TL_DEBUG_OK(ok, TL_DEBUG_TOKEN, id);  // (an id outside the vocabulary reads as a zero row)
  if (pairs && threadIdx.x == 0) {
    const int req = token_req[t], first = req_indptr[req];
    int previous = 0;
    if (t > first) {
      previous = ids[t - 1];
    } else {
      const int slot = slots[req];
      if (TL_DEBUG_OK(slot >= -1 && slot < max_slots, TL_DEBUG_SLOT, slot) && slot >= 0 && slot < max_slots) {
        previous = last[slot];
        last[slot] = ids[req_indptr[req + 1] - 1];
      }
    }
    long long row = (previous * mul_prev + id * mul_cur) % buckets;
    if (row < 0) row += buckets;
    pair_row = positions[t] == 0 ? (long long)buckets : row;
  }
  __syncthreads();
  const T* row = table + (size_t)(ok ? id : 0) * width;
  const T* pair = pairs ? pairs + (size_t)pair_row * width : nullptr;
  float sum = 0.f;
  for (int c = threadIdx.x; c < width; c += NT) {
    float v = ok ? to_float(row[c]) * scale : 0.f;
    if (pair) v += to_float(pair[c]);
    x[c] = v;
    sum += v;
  }
  float mean = 0.f, inv = 1.f;
  if (weight) {
    if (centre) mean = block_sum<NT>(sum, scratch) / (float)width;
    float ss = 0.f;
    for (int c = threadIdx.x; c < width; c += NT) {  // a thread reads back what it wrote itself
      const float d = x[c] - mean;
      ss = fmaf(d, d, ss);
    }
    inv = 1.f / sqrtf(block_sum<NT>(ss, scratch) / (float)width + eps);
  }
  float* o = out + (size_t)t * streams * width;
  for (int c = threadIdx.x; c < width; c += NT) {
    float v = x[c];
    if (weight) {
      v = (v - mean) * inv * weight[c];
      if (bias) v += bias[c];
    }
    for (int s = 0; s < streams; ++s) o[(size_t)s * width + c] = v;
  }
}

}  // namespace

TL_DEBUG_READER(tl_token_embed_debug_error)

// table [vocab, width]; pairs (or null) [buckets + 1, width] of the same type; out float32 [tokens, streams, width].
extern "C" int tl_token_embed(const void* table, const void* pairs, int dtype, const int* ids, const int* positions,
                              const int* token_req, const int* req_indptr, const int* slots, int* last, int max_slots,
                              int buckets, long long mul_prev, long long mul_cur, const float* weight, const float* bias,
                              float eps, int centre, float* out, int tokens, int streams, int width, int vocab, float scale,
                              cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (streams <= 0 || width <= 0 || (size_t)width * sizeof(float) > 200 * 1024) return TL_ERR_UNSUPPORTED;
  if (pairs && (buckets <= 0 || !positions || !token_req || !req_indptr || !slots || !last)) return TL_ERR_UNSUPPORTED;
  const size_t smem = (size_t)width * sizeof(float);
  auto run = [&](auto kernel, auto* typed, auto* typed_pairs) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    tl::launch_kernel(kernel, (unsigned)tokens, NT, smem, stream, typed, typed_pairs, ids, positions, token_req, req_indptr,
                      slots, last, max_slots, buckets, mul_prev, mul_cur, weight, bias, eps, centre, out, streams, width,
                      vocab, scale);
  };
  if (dtype == TL_DTYPE_F32) run(token_embed_kernel<float>, (const float*)table, (const float*)pairs);
  else run(token_embed_kernel<__nv_bfloat16>, (const __nv_bfloat16*)table, (const __nv_bfloat16*)pairs);
  return TL_LAUNCH_CHECK();
}
