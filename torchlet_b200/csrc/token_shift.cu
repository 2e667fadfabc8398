// The token shift in front of a time-mixing recurrence: several mixes of a token's row with the row before it,
//
//   out[c][t] = x[t] + (x[t - 1] - x[t]) * mu[c]        c = 0 .. n - 1, element by element, float32 inside,
//
// along each request's tokens.  The row before a request's first token of the step is the slot's row of ``state``
// [slots][width] (float32; zeros at a sequence's start, which is what a cleared slot holds).  The block of that first
// token also moves the request's LAST row of the step into the slot: the thread that owns a channel reads the old
// number before it writes the new one, so one kernel does both whatever the portion's length.
// out: [n][plane] with rows of ``width``, in the type of x; plane >= tokens * width.
#include "common.cuh"

namespace {

using namespace tl;

constexpr int NT = 128;

template <int V> __device__ __forceinline__ void load_row(const float* p, float (&v)[V]) {
#pragma unroll
  for (int j = 0; j < V; ++j) v[j] = p[j];
}
template <int V> __device__ __forceinline__ void load_row(const __nv_bfloat16* p, float (&v)[V]) {
  if constexpr (V == 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(raw.x << 16);
    v[1] = __uint_as_float(raw.x & 0xffff0000u);
    v[2] = __uint_as_float(raw.y << 16);
    v[3] = __uint_as_float(raw.y & 0xffff0000u);
  } else {
    v[0] = __bfloat162float(*p);
  }
}
template <int V> __device__ __forceinline__ void load_wide(const float* p, float (&v)[V]) {
  if constexpr (V == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
  } else {
    v[0] = *p;
  }
}
template <int V> __device__ __forceinline__ void store_row(float* p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int V> __device__ __forceinline__ void store_row(__nv_bfloat16* p, const float (&v)[V]) {
  if constexpr (V == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
  } else {
    *p = __float2bfloat16_rn(v[0]);
  }
}

// grid: (tokens, channel blocks of NT * V); a thread owns V neighbouring channels of one token.
template <typename T, int V>
__global__ void __launch_bounds__(NT)
token_shift_kernel(const T* __restrict__ x, const float* __restrict__ mu, int n, T* __restrict__ out, long long plane,
                   float* __restrict__ state, int max_slots, const int* __restrict__ token_req,
                   const int* __restrict__ req_indptr, const int* __restrict__ slots, int width) {
  tl::pdl_launch_dependents();
  tl::pdl_wait();
  const int t = blockIdx.x;
  const int c = (blockIdx.y * NT + threadIdx.x) * V;
  if (c >= width) return;
  const int req = token_req[t];
  const int first = req_indptr[req];
  float now[V], before[V];
  load_row<V>(x + (size_t)t * width + c, now);
#pragma unroll
  for (int j = 0; j < V; ++j) before[j] = 0.f;
  if (t > first) {
    load_row<V>(x + (size_t)(t - 1) * width + c, before);
  } else {
    const int slot = slots[req];
    if (TL_DEBUG_OK(slot >= -1 && slot < max_slots, TL_DEBUG_SLOT, slot) && slot >= 0) {
      float* mine = state + (size_t)slot * width + c;
      float last[V];
      load_row<V>(x + (size_t)(req_indptr[req + 1] - 1) * width + c, last);
      load_wide<V>(mine, before);
      store_row<V>(mine, last);
    }
  }
  for (int k = 0; k < n; ++k) {
    float m[V], v[V];
    load_wide<V>(mu + (size_t)k * width + c, m);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = fmaf(before[j] - now[j], m[j], now[j]);
    store_row<V>(out + (size_t)k * plane + (size_t)t * width + c, v);
  }
}

}  // namespace

TL_DEBUG_READER(tl_token_shift_debug_error)

extern "C" int tl_token_shift(const void* x, int dtype, const float* mu, int n, void* out, long long plane, float* state,
                              int max_slots, const int* token_req, const int* req_indptr, const int* slots, int requests,
                              int tokens, int width, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (n <= 0 || width <= 0 || requests <= 0 || plane < (long long)tokens * width) return TL_ERR_UNSUPPORTED;
  const uintptr_t all = (uintptr_t)x | (uintptr_t)mu | (uintptr_t)out | (uintptr_t)state;
  const bool wide = width % 4 == 0 && plane % 4 == 0 && (all & 15) == 0;
  const int per = NT * (wide ? 4 : 1);
  const dim3 grid(tokens, (width + per - 1) / per);
  if (grid.y > 65535) return TL_ERR_UNSUPPORTED;
#define TL_SHIFT(T, V)                                                                                             \
  tl::launch_kernel(token_shift_kernel<T, V>, grid, NT, 0, stream, (const T*)x, mu, n, (T*)out, plane, state, max_slots, \
                    token_req, req_indptr, slots, width)
  if (dtype == TL_DTYPE_F32) {
    if (wide) TL_SHIFT(float, 4);
    else TL_SHIFT(float, 1);
  } else {
    if (wide) TL_SHIFT(__nv_bfloat16, 4);
    else TL_SHIFT(__nv_bfloat16, 1);
  }
#undef TL_SHIFT
  return TL_LAUNCH_CHECK();
}
