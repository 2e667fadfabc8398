// What stands between the q/k/v product and the paged attention of a mixer whose scores are MIXED ACROSS THE HEADS
// before the softmax, whose key and value sizes may differ, and whose values may be mixed with an earlier layer's.
// One block per token; everything float32 until the stores.  The projections arrive as float32 rows
//   [ q (H D) | k (G D) | v (G V) ]
// either finished, or as the split sums a product left ([splits][tokens][row]) with the biases still to be added.
//
//   q <- q / rms(q over all H D) * wq,  k <- k / rms(k over all G D) * wk      (``wq`` / ``wk`` null: no norm)
//   the first ``dims`` entries of every head of q and k turn by the token's position, entry i with i + dims / 2
//   v <- (1 - l) v + l v_first            (``value_mode`` 2; with mode 1 this layer's v is written to ``v_first``)
//   k and v go to the token's cache row, padded with zeros to P entries each
//
// Mixed scores, s'_h = sum_g M[h, g] s_g with s_g = q_g . k_(g's KV head), are linear in the queries: with the query of
// head h SPREAD over all KV heads,
//   q'_h = [ sum over the heads g of KV head c of M[h, g] q_g ]  for c = 0 .. G - 1,        s'_h = q'_h . [k_0 .. k_(G-1)]
// ``spread`` 1 writes q' rows [H][G][P]; 0 writes the queries themselves, [H][P] at the start of the row (for a kernel
// that mixes the scores it has computed); 2 writes q' for the tokens of requests that bring several tokens and q for
// single tokens.  Without a matrix (``mix`` null) rows are always [H][P].
#include <math.h>

#include "common.cuh"

namespace {

using namespace tl;

constexpr int NT = 256;

struct Params {
  const float* src;  // [splits][tokens][src_stride]
  int splits;
  long long split_stride;
  int src_stride;
  const float *bias, *wq, *wk, *inv_freq;
  float magnitude, eps;
  const int *positions, *token_req, *req_indptr, *block_table;
  int table_width, page_size, num_pages;
  int H, G, D, V, P, dims;
  const float* mix;  // [H][H] or null
  int spread;
  float* v_first;  // [tokens][G V]
  const float* lambda;
  int value_mode;  // 0: none; 1: this layer's values are the first ones; 2: mixed with the first ones
  int write_kv;
  long long q_stride;
};

template <typename T> __device__ __forceinline__ void store2(T* p, float a, float b);
template <> __device__ __forceinline__ void store2<float>(float* p, float a, float b) {
  *reinterpret_cast<float2*>(p) = make_float2(a, b);
}
template <> __device__ __forceinline__ void store2<__nv_bfloat16>(__nv_bfloat16* p, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}

// q' of one token; ``PER`` = H / G query heads a KV head where that is 1, 2, 4 or 8 (their entries then stay in
// registers for all H rows), else 0.
template <typename T, int PER>
__device__ __forceinline__ void spread_queries(const Params& p, const float* q, const float* mix, T* out) {
  const int per = PER > 0 ? PER : p.H / p.G;
  const int pairs = p.P >> 1, items = p.G * pairs;
  const int rows = max(1, min(p.H, NT / max(1, items)));  // threads that share a column pair, each with its own heads
  for (int item = threadIdx.x; item < items * rows; item += NT) {
    const int col = item % items, part = item / items;
    const int c = col / pairs, i = (col - c * pairs) * 2;
    const bool in0 = i < p.D, in1 = i + 1 < p.D;
    const float* base = q + (size_t)c * per * p.D + i;
    float v0[PER > 0 ? PER : 1], v1[PER > 0 ? PER : 1];
    if constexpr (PER > 0) {
#pragma unroll
      for (int j = 0; j < PER; ++j) {
        v0[j] = in0 ? base[j * p.D] : 0.f;
        v1[j] = in1 ? base[j * p.D + 1] : 0.f;
      }
    }
    for (int h = part; h < p.H; h += rows) {
      const float* m = mix + h * p.H + c * per;
      float a = 0.f, b = 0.f;
      if constexpr (PER > 0) {
#pragma unroll
        for (int j = 0; j < PER; ++j) {
          a = fmaf(m[j], v0[j], a);
          b = fmaf(m[j], v1[j], b);
        }
      } else {
        for (int j = 0; j < per; ++j) {
          a = fmaf(m[j], in0 ? base[j * p.D] : 0.f, a);
          b = fmaf(m[j], in1 ? base[j * p.D + 1] : 0.f, b);
        }
      }
      store2<T>(out + ((size_t)h * p.G + c) * p.P + i, a, b);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(NT)
qkv_prepare_kernel(const Params p, T* __restrict__ pages, T* __restrict__ q_out) {
  tl::pdl_launch_dependents();
  tl::pdl_wait();
  extern __shared__ __align__(16) float smem[];
  __shared__ float scratch[32];
  const int t = blockIdx.x;
  const int qn = p.H * p.D, kn = p.G * p.D, vn = p.G * p.V, half = p.dims >> 1;
  float* q = smem;            // H D
  float* k = q + qn;          // G D
  float* v = k + kn;          // G V
  float* cosines = v + vn;    // half
  float* sines = cosines + half;
  float* mix = sines + half;  // H H
  const int pos = p.positions[t];
  const int req = p.token_req[t];
  const bool spread = p.mix && (p.spread == 1 || (p.spread == 2 && p.req_indptr[req + 1] - p.req_indptr[req] > 1));
  for (int i = threadIdx.x; i < half; i += NT) {
    float sn, cs;
    sincosf((float)pos * p.inv_freq[i], &sn, &cs);
    cosines[i] = cs * p.magnitude;
    sines[i] = sn * p.magnitude;
  }
  if (spread)
    for (int i = threadIdx.x; i < p.H * p.H; i += NT) mix[i] = p.mix[i];
  const float* row = p.src + (size_t)t * p.src_stride;
  float ssq = 0.f, ssk = 0.f;
  for (int i = threadIdx.x; i < qn + kn + vn; i += NT) {
    float x = 0.f;
    for (int s = 0; s < p.splits; ++s) x += row[(size_t)s * p.split_stride + i];
    if (p.bias) x += p.bias[i];
    smem[i] = x;
    if (i < qn) ssq = fmaf(x, x, ssq);
    else if (i < qn + kn) ssk = fmaf(x, x, ssk);
  }
  const float inv_q = p.wq ? 1.f / sqrtf(block_sum<NT>(ssq, scratch) / (float)qn + p.eps) : 1.f;
  const float inv_k = p.wk ? 1.f / sqrtf(block_sum<NT>(ssk, scratch) / (float)kn + p.eps) : 1.f;
  __syncthreads();
  // norm and rotation, in place: the lower entry of a rotated pair does both
  const int per_head = half + (p.D - p.dims);
  for (int item = threadIdx.x; item < (p.H + p.G) * per_head; item += NT) {
    const int head = item / per_head, i = item - head * per_head;
    const int e = i < half ? i : i + half;
    float* x = smem + (size_t)head * p.D + e;
    const bool is_q = head < p.H;
    const float* w = is_q ? p.wq : p.wk;
    if (w) w += (size_t)(is_q ? head : head - p.H) * p.D + e;
    const float inv = is_q ? inv_q : inv_k;
    const float a = x[0] * inv * (w ? w[0] : 1.f);
    if (i < half) {
      const float b = x[half] * inv * (w ? w[half] : 1.f);
      x[0] = a * cosines[i] - b * sines[i];
      x[half] = b * cosines[i] + a * sines[i];
    } else {
      x[0] = a;
    }
  }
  if (p.value_mode == 1) {
    for (int i = threadIdx.x; i < vn; i += NT) p.v_first[(size_t)t * vn + i] = v[i];
  } else if (p.value_mode == 2) {
    const float l = *p.lambda;
    for (int i = threadIdx.x; i < vn; i += NT) v[i] = (1.f - l) * v[i] + l * p.v_first[(size_t)t * vn + i];
  }
  __syncthreads();
  const int pairs = p.P >> 1;
  if (p.write_kv) {
    int page = -1;
    if (TL_DEBUG_OK(pos / p.page_size < p.table_width, TL_DEBUG_POSITION, pos))
      page = p.block_table[(size_t)req * p.table_width + pos / p.page_size];
    if (TL_DEBUG_OK(page >= 0 && page < p.num_pages, TL_DEBUG_PAGE, page) && page >= 0) {
      // pages: [num_pages, 2, G, page_size, P]
      T* dst = pages + (size_t)page * 2 * p.G * p.page_size * p.P + (size_t)(pos % p.page_size) * p.P;
      for (int item = threadIdx.x; item < 2 * p.G * pairs; item += NT) {
        const int head = item / pairs, i = (item - head * pairs) * 2;  // key heads, then value heads
        const bool is_v = head >= p.G;
        const int n = is_v ? p.V : p.D;
        const float* src = is_v ? v + (size_t)(head - p.G) * p.V : k + (size_t)head * p.D;
        store2<T>(dst + (size_t)head * p.page_size * p.P + i, i < n ? src[i] : 0.f, i + 1 < n ? src[i + 1] : 0.f);
      }
    }
  }
  T* out = q_out + (size_t)t * p.q_stride;
  if (!spread) {
    for (int item = threadIdx.x; item < p.H * pairs; item += NT) {
      const int head = item / pairs, i = (item - head * pairs) * 2;
      const float* src = q + (size_t)head * p.D;
      store2<T>(out + (size_t)head * p.P + i, i < p.D ? src[i] : 0.f, i + 1 < p.D ? src[i + 1] : 0.f);
    }
    return;
  }
  switch (p.H / p.G) {
    case 1: spread_queries<T, 1>(p, q, mix, out); break;
    case 2: spread_queries<T, 2>(p, q, mix, out); break;
    case 4: spread_queries<T, 4>(p, q, mix, out); break;
    case 8: spread_queries<T, 8>(p, q, mix, out); break;
    default: spread_queries<T, 0>(p, q, mix, out); break;
  }
}

template <typename T>
int launch(const Params& p, void* pages, void* q_out, int tokens, cudaStream_t stream) {
  const size_t floats = (size_t)p.H * p.D + (size_t)p.G * (p.D + p.V) + p.dims + (p.mix ? (size_t)p.H * p.H : 0);
  const size_t smem = floats * sizeof(float);
  if (smem > 200 * 1024) return TL_ERR_UNSUPPORTED;
  if (smem > 48 * 1024) {
    const cudaError_t err = cudaFuncSetAttribute(qkv_prepare_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
  }
  tl::launch_kernel(qkv_prepare_kernel<T>, (unsigned)tokens, NT, smem, stream, p, (T*)pages, (T*)q_out);
  return TL_LAUNCH_CHECK();
}

}  // namespace

TL_DEBUG_READER(tl_qkv_prepare_debug_error)

// src: finished rows (splits 1) or split sums; bias: null, or still to be added (H D + G D + G V floats).
// pages: one cache layer [num_pages][2][G][page_size][P]; P even, at least D and V.  q_out rows of q_stride elements.
extern "C" int tl_qkv_prepare(const float* src, int splits, long long split_stride, int src_stride, const float* bias,
                              const float* wq, const float* wk, const float* inv_freq, float magnitude, float eps,
                              const int* positions, const int* token_req, const int* req_indptr, const int* block_table,
                              int table_width, void* pages, int dtype, int page_size, int num_pages, void* q_out,
                              long long q_stride, int tokens, int H, int G, int D, int V, int P, int dims,
                              const float* mix, int spread, float* v_first, const float* lambda, int value_mode,
                              int write_kv, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || V <= 0 || P < D || P < V || P % 2 || q_stride % 2 || page_size <= 0 || splits < 1)
    return TL_ERR_UNSUPPORTED;
  if (dims < 0 || dims % 2 || dims > D || (dims && !inv_freq)) return TL_ERR_UNSUPPORTED;
  if (value_mode < 0 || value_mode > 2 || (value_mode && !v_first) || (value_mode == 2 && !lambda)) return TL_ERR_UNSUPPORTED;
  if (spread < 0 || spread > 2 || (spread == 2 && !req_indptr)) return TL_ERR_UNSUPPORTED;
  if (q_stride < (long long)H * P * (mix && spread ? G : 1)) return TL_ERR_UNSUPPORTED;
  Params p;
  p.src = src; p.splits = splits; p.split_stride = split_stride; p.src_stride = src_stride;
  p.bias = bias; p.wq = wq; p.wk = wk; p.inv_freq = inv_freq; p.magnitude = magnitude; p.eps = eps;
  p.positions = positions; p.token_req = token_req; p.req_indptr = req_indptr; p.block_table = block_table;
  p.table_width = table_width; p.page_size = page_size; p.num_pages = num_pages;
  p.H = H; p.G = G; p.D = D; p.V = V; p.P = P; p.dims = dims;
  p.mix = mix; p.spread = spread; p.v_first = v_first; p.lambda = lambda; p.value_mode = value_mode;
  p.write_kv = write_kv; p.q_stride = q_stride;
  return dtype == TL_DTYPE_F32 ? launch<float>(p, pages, q_out, tokens, stream)
                               : launch<__nv_bfloat16>(p, pages, q_out, tokens, stream);
}
