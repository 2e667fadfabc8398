// The end of a sub-layer whose OUTPUT is normed, and the start of the next one, in one pass over the rows (float32):
//
//   v = y (+ partial sums of y's last product) (+ its bias)            a sub-layer's output
//   v *= sigmoid(g),  g = the gate's row (or its partial sums) + bias  (optional)
//   acc += m * norm(v) (+ row)                                         norm: layer norm or RMS norm, weight (and bias)
//   out = norm'(acc) in the compute type                               (optional) what the next sub-layer reads
//
// A row is kept in registers from the first load to the last store: one trip to memory, four block sums.  Without split
// sums (the 32-bit engine has none) the order of the additions depends on the width alone.  ``y`` may be left zeroed for the next sub-layer to add into.
//
//   add_row        acc[t] += row for every token
//   relu_squared   x = max(x, 0)^2 in place (where the product before it has no such epilogue)
#include <math.h>

#include "common.cuh"

namespace {

using namespace tl;

struct Args {
  float* acc;
  float* y;
  const float* partials;  // [splits][rows][width]
  const float* y_bias;
  const float* gate;      // [gate_splits][rows][width], or null
  const float* gate_bias;
  const float* weight;
  const float* bias;
  const float* row;
  void* out;
  const float* weight2;
  const float* bias2;
  float eps, m, eps2;
  int splits, gate_splits, centre, centre2, width, clear;
  size_t plane;           // rows * width
};

template <int V> __device__ __forceinline__ void load_v(const float* p, float (&out)[V]) {
  if constexpr (V == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    out[0] = v.x; out[1] = v.y; out[2] = v.z; out[3] = v.w;
  } else {
    out[0] = *p;
  }
}
template <int V> __device__ __forceinline__ void store_v(float* p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int V> __device__ __forceinline__ void store_v(__nv_bfloat16* p, const float (&v)[V]) {
  if constexpr (V == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
  } else {
    *p = __float2bfloat16_rn(v[0]);
  }
}

// sum += the ``count`` planes of src at the thread's entries, in ascending order, all of eight planes' loads of an entry
// in flight: a step of few tokens is a chain of dependent trips to memory.
template <int NT, int PER, int V>
__device__ __forceinline__ void add_planes(float (&sum)[PER][V], const float* src, int count, size_t plane, int width) {
  constexpr int BATCH = 8;
  for (int s0 = 0; s0 < count; s0 += BATCH) {
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      const int j = (threadIdx.x + k * NT) * V;
      if (j < width) {
        float part[BATCH][V];
#pragma unroll
        for (int s = 0; s < BATCH; ++s) {
#pragma unroll
          for (int e = 0; e < V; ++e) part[s][e] = 0.f;
          if (s0 + s < count) load_v<V>(src + (s0 + s) * plane + j, part[s]);
        }
#pragma unroll
        for (int s = 0; s < BATCH; ++s)
#pragma unroll
          for (int e = 0; e < V; ++e) sum[k][e] += part[s][e];
      }
    }
  }
}

// The mean (0 without centring) and 1 / sqrt(variance + eps) of the row the threads hold; entries past the width are 0.
template <int NT, int PER, int V>
__device__ __forceinline__ float2 moments(const float (&v)[PER][V], int width, float eps, int centre, float* scratch) {
  float mean = 0.f;
  if (centre) {
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < PER; ++k)
#pragma unroll
      for (int e = 0; e < V; ++e) sum += v[k][e];
    mean = block_sum<NT>(sum, scratch) / (float)width;
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    if ((threadIdx.x + k * NT) * V < width) {
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float d = v[k][e] - mean;
        ss = fmaf(d, d, ss);
      }
    }
  }
  return make_float2(mean, 1.f / sqrtf(block_sum<NT>(ss, scratch) / (float)width + eps));
}

// One block a row; a thread holds PER x V entries of it.  SUMS: y or the gate comes with split sums.
template <typename T, int NT, int PER, int V, bool SUMS>
__global__ void __launch_bounds__(NT)
residual_norm_kernel(const Args a) {
  tl::pdl_launch_dependents();
  __shared__ float scratch[32];
  // the weights are written by no kernel: asked for before the wait on the preceding one
  float w[PER][V], w2[PER][V];
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int j = (threadIdx.x + k * NT) * V;
    if (j < a.width) {
      load_v<V>(a.weight + j, w[k]);
      if (a.out) load_v<V>(a.weight2 + j, w2[k]);
    }
  }
  tl::pdl_wait();
  const size_t at = (size_t)blockIdx.x * a.width;
  float v[PER][V], x[PER][V], g[PER][V];
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int j = (threadIdx.x + k * NT) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) v[k][e] = x[k][e] = g[k][e] = 0.f;
    if (j < a.width) {
      load_v<V>(a.y + at + j, v[k]);
      load_v<V>(a.acc + at + j, x[k]);
      if (a.gate) load_v<V>(a.gate + at + j, g[k]);
    }
  }
  if constexpr (SUMS) {
    add_planes<NT, PER, V>(v, a.partials + at, a.splits, a.plane, a.width);
    if (a.gate) add_planes<NT, PER, V>(g, a.gate + a.plane + at, a.gate_splits - 1, a.plane, a.width);
  }
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int j = (threadIdx.x + k * NT) * V;
    if (j < a.width) {
      if (a.y_bias) {
        float b[V];
        load_v<V>(a.y_bias + j, b);
#pragma unroll
        for (int e = 0; e < V; ++e) v[k][e] += b[e];
      }
      if (a.gate) {
        if (a.gate_bias) {
          float b[V];
          load_v<V>(a.gate_bias + j, b);
#pragma unroll
          for (int e = 0; e < V; ++e) g[k][e] += b[e];
        }
#pragma unroll
        for (int e = 0; e < V; ++e) v[k][e] *= 1.f / (1.f + expf(-g[k][e]));
      }
    }
  }
  const float2 first = moments<NT, PER, V>(v, a.width, a.eps, a.centre, scratch);
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int j = (threadIdx.x + k * NT) * V;
    if (j < a.width) {
      float add[V];
#pragma unroll
      for (int e = 0; e < V; ++e) add[e] = (v[k][e] - first.x) * first.y * w[k][e];
      if (a.bias) {
        float b[V];
        load_v<V>(a.bias + j, b);
#pragma unroll
        for (int e = 0; e < V; ++e) add[e] += b[e];
      }
#pragma unroll
      for (int e = 0; e < V; ++e) x[k][e] = fmaf(a.m, add[e], x[k][e]);
      if (a.row) {
        float r[V];
        load_v<V>(a.row + j, r);
#pragma unroll
        for (int e = 0; e < V; ++e) x[k][e] += r[e];
      }
      store_v<V>(a.acc + at + j, x[k]);
      if (a.clear) {
        float zero[V];
#pragma unroll
        for (int e = 0; e < V; ++e) zero[e] = 0.f;
        store_v<V>(a.y + at + j, zero);
      }
    }
  }
  if (!a.out) return;
  const float2 second = moments<NT, PER, V>(x, a.width, a.eps2, a.centre2, scratch);
  T* out = reinterpret_cast<T*>(a.out) + at;
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int j = (threadIdx.x + k * NT) * V;
    if (j < a.width) {
      float o[V];
#pragma unroll
      for (int e = 0; e < V; ++e) o[e] = (x[k][e] - second.x) * second.y * w2[k][e];
      if (a.bias2) {
        float b[V];
        load_v<V>(a.bias2 + j, b);
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] += b[e];
      }
      store_v<V>(out + j, o);
    }
  }
}

template <typename T>
int launch_residual(const Args& a, int rows, cudaStream_t stream) {
  const uintptr_t all = (uintptr_t)a.acc | (uintptr_t)a.y | (uintptr_t)a.partials | (uintptr_t)a.y_bias | (uintptr_t)a.gate |
                        (uintptr_t)a.gate_bias | (uintptr_t)a.weight | (uintptr_t)a.bias | (uintptr_t)a.row |
                        (uintptr_t)a.out | (uintptr_t)a.weight2 | (uintptr_t)a.bias2;
  const bool wide = a.width % 4 == 0 && (all & 15) == 0;
  const bool sums = a.splits > 0 || (a.gate && a.gate_splits > 1);
#define TL_RESIDUAL(NT, PER, V)                                                                               \
  {                                                                                                           \
    if (sums) tl::launch_kernel(residual_norm_kernel<T, NT, PER, V, true>, (unsigned)rows, NT, 0, stream, a); \
    else tl::launch_kernel(residual_norm_kernel<T, NT, PER, V, false>, (unsigned)rows, NT, 0, stream, a);     \
  }
  if (wide && sums && a.width <= 4096 && rows <= 512) {  // few rows: one round of loads a thread
    if (a.width <= 1024) TL_RESIDUAL(256, 1, 4)
    else if (a.width <= 2048) TL_RESIDUAL(512, 1, 4)
    else TL_RESIDUAL(1024, 1, 4)
  } else if (wide) {
    if (a.width <= 1024) TL_RESIDUAL(256, 1, 4)
    else if (a.width <= 2048) TL_RESIDUAL(256, 2, 4)
    else if (a.width <= 4096) TL_RESIDUAL(512, 2, 4)
    else if (a.width <= 8192) TL_RESIDUAL(512, 4, 4)
    else if (a.width <= 16384) TL_RESIDUAL(1024, 4, 4)
    else return TL_ERR_UNSUPPORTED;
  } else {
    if (a.width <= 1024) TL_RESIDUAL(256, 4, 1)
    else if (a.width <= 4096) TL_RESIDUAL(512, 8, 1)
    else if (a.width <= 16384) TL_RESIDUAL(1024, 16, 1)
    else return TL_ERR_UNSUPPORTED;
  }
#undef TL_RESIDUAL
  return TL_LAUNCH_CHECK();
}

__global__ void add_row_kernel(float* __restrict__ acc, const float* __restrict__ row, int width, size_t total) {
  tl::pdl_launch_dependents();
  tl::pdl_wait();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < total) acc[i] += row[i % width];
}

template <typename T>
__global__ void relu_squared_kernel(T* __restrict__ x, size_t total) {
  tl::pdl_launch_dependents();
  tl::pdl_wait();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const float r = fmaxf(to_float(x[i]), 0.f);
  x[i] = from_float<T>(r * r);
}

}  // namespace

extern "C" {

// acc, y float32 [rows][width]; partials [splits][rows][width] (splits 0: none); gate [gate_splits][rows][width] or null;
// centre: layer norm, else RMS norm; row, out (with weight2 ...) and the biases may be null.  width up to 16,384.
int tl_residual_norm(float* acc, float* y, const float* partials, int splits, const float* y_bias, const float* gate,
                     int gate_splits, const float* gate_bias, const float* weight, const float* bias, float eps,
                     int centre, float m, const float* row, void* out, int out_dtype, const float* weight2,
                     const float* bias2, float eps2, int centre2, int rows, int width, int clear, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (width <= 0 || splits < 0 || (splits && !partials) || gate_splits < 1 || (out && !weight2)) return TL_ERR_UNSUPPORTED;
  Args a;
  a.acc = acc;
  a.y = y;
  a.partials = partials;
  a.y_bias = y_bias;
  a.gate = gate;
  a.gate_bias = gate_bias;
  a.weight = weight;
  a.bias = bias;
  a.row = row;
  a.out = out;
  a.weight2 = weight2;
  a.bias2 = bias2;
  a.eps = eps;
  a.m = m;
  a.eps2 = eps2;
  a.splits = splits;
  a.gate_splits = gate_splits;
  a.centre = centre;
  a.centre2 = centre2;
  a.width = width;
  a.clear = clear;
  a.plane = (size_t)rows * width;
  return out_dtype == TL_DTYPE_F32 ? launch_residual<float>(a, rows, stream) : launch_residual<__nv_bfloat16>(a, rows, stream);
}

int tl_add_row(float* acc, const float* row, int rows, int width, cudaStream_t stream) {
  const size_t total = (size_t)rows * width;
  if (total == 0) return 0;
  tl::launch_kernel(add_row_kernel, (unsigned)((total + 255) / 256), 256, 0, stream, acc, row, width, total);
  return TL_LAUNCH_CHECK();
}

int tl_relu_squared(void* x, int dtype, long long n, cudaStream_t stream) {
  if (n <= 0) return 0;
  const unsigned blocks = (unsigned)((n + 255) / 256);
  if (dtype == TL_DTYPE_F32)
    tl::launch_kernel(relu_squared_kernel<float>, blocks, 256, 0, stream, (float*)x, (size_t)n);
  else
    tl::launch_kernel(relu_squared_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (__nv_bfloat16*)x, (size_t)n);
  return TL_LAUNCH_CHECK();
}

}  // extern "C"
