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

// V consecutive channels: 4 where width and addresses allow 16-byte pieces (8-byte ones of the bfloat16 tables), else 1.
template <int V> __device__ __forceinline__ void load_v(const float* p, float (&out)[V]) {
  if constexpr (V == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    out[0] = v.x; out[1] = v.y; out[2] = v.z; out[3] = v.w;
  } else {
    out[0] = *p;
  }
}
template <int V> __device__ __forceinline__ void load_v(const __nv_bfloat16* p, float (&out)[V]) {
  if constexpr (V == 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    out[0] = __uint_as_float(raw.x << 16);
    out[1] = __uint_as_float(raw.x & 0xffff0000u);
    out[2] = __uint_as_float(raw.y << 16);
    out[3] = __uint_as_float(raw.y & 0xffff0000u);
  } else {
    out[0] = __bfloat162float(*p);
  }
}
template <int V> __device__ __forceinline__ void store_v(float* p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}

template <typename T, int V>
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
  for (int c = threadIdx.x * V; c < width; c += NT * V) {
    float v[V];
    load_v<V>(row + c, v);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = ok ? v[e] * scale : 0.f;
    if (pair) {
      float w[V];
      load_v<V>(pair + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += w[e];
    }
    store_v<V>(x + c, v);
#pragma unroll
    for (int e = 0; e < V; ++e) sum += v[e];
  }
  float mean = 0.f, inv = 1.f;
  if (weight) {
    if (centre) mean = block_sum<NT>(sum, scratch) / (float)width;
    float ss = 0.f;
    for (int c = threadIdx.x * V; c < width; c += NT * V) {  // a thread reads back what it wrote itself
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float d = x[c + e] - mean;
        ss = fmaf(d, d, ss);
      }
    }
    inv = 1.f / sqrtf(block_sum<NT>(ss, scratch) / (float)width + eps);
  }
  float* o = out + (size_t)t * streams * width;
  for (int c = threadIdx.x * V; c < width; c += NT * V) {
    float v[V];
    load_v<V>(x + c, v);
    if (weight) {
      float w[V];
      load_v<V>(weight + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = (v[e] - mean) * inv * w[e];
      if (bias) {
        load_v<V>(bias + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] += w[e];
      }
    }
    for (int s = 0; s < streams; ++s) store_v<V>(o + (size_t)s * width + c, v);
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
  const uintptr_t all = (uintptr_t)table | (uintptr_t)pairs | (uintptr_t)weight | (uintptr_t)bias | (uintptr_t)out;
  const bool wide = width % 4 == 0 && (all & 15) == 0;
  const float *table32 = (const float*)table, *pairs32 = (const float*)pairs;
  const __nv_bfloat16 *table16 = (const __nv_bfloat16*)table, *pairs16 = (const __nv_bfloat16*)pairs;
  if (dtype == TL_DTYPE_F32) {
    if (wide) run(token_embed_kernel<float, 4>, table32, pairs32);
    else run(token_embed_kernel<float, 1>, table32, pairs32);
  } else {
    if (wide) run(token_embed_kernel<__nv_bfloat16, 4>, table16, pairs16);
    else run(token_embed_kernel<__nv_bfloat16, 1>, table16, pairs16);
  }
  return TL_LAUNCH_CHECK();
}
