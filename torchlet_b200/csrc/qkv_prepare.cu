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
  int mix_floats;    // shared memory it takes
  int spread;
  float* v_first;  // [tokens][G V]
  const float* lambda;
  int value_mode;  // 0: none; 1: this layer's values are the first ones; 2: mixed with the first ones
  int write_kv;
  long long q_stride;
};

// W consecutive floats (4 where every size and address allows 16-byte pieces, else 1).
template <int W> __device__ __forceinline__ void load_w(const float* p, float (&v)[W]) {
  if constexpr (W == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
  } else {
    v[0] = *p;
  }
}
template <int W> __device__ __forceinline__ void store_w(float* p, const float (&v)[W]) {
  if constexpr (W == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int W> __device__ __forceinline__ void store_w(__nv_bfloat16* p, const float (&v)[W]) {
  if constexpr (W == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
  } else {
    *p = __float2bfloat16_rn(v[0]);
  }
}

// q' of one token; ``PER`` = H / G query heads a KV head where that is 1, 2, 4 or 8 (their entries then stay in
// registers for all H rows), else 0.
template <typename T, int NT, int PER, int W>
__device__ __forceinline__ void spread_queries(const Params& p, const float* q, const float* mix, T* out) {
  const int per = PER > 0 ? PER : p.H / p.G;
  const int pieces = p.P / W, items = p.G * pieces;
  const int rows = max(1, min(p.H, NT / max(1, items)));  // threads that share a column piece, each with its own heads
  for (int item = threadIdx.x; item < items * rows; item += NT) {
    const int part = item / items, col = item - part * items;
    const int c = col / pieces, i = (col - c * pieces) * W;
    const bool in = i < p.D;
    const float* base = q + (size_t)c * per * p.D + (in ? i : 0);
    float v[PER > 0 ? PER : 1][W];
    if constexpr (PER > 0) {
#pragma unroll
      for (int j = 0; j < PER; ++j) {
        load_w<W>(base + j * p.D, v[j]);
        if (!in)
#pragma unroll
          for (int e = 0; e < W; ++e) v[j][e] = 0.f;
      }
    }
    for (int h = part; h < p.H; h += rows) {
      const float* m = mix + h * p.H + c * per;
      float sum[W];
#pragma unroll
      for (int e = 0; e < W; ++e) sum[e] = 0.f;
      if constexpr (PER > 0) {
        float f[PER];
        if constexpr (PER % 4 == 0) {  // (rows of the matrix then start on 16-byte boundaries)
#pragma unroll
          for (int j = 0; j < PER; j += 4) load_w<4>(m + j, reinterpret_cast<float(&)[4]>(f[j]));
        } else {
#pragma unroll
          for (int j = 0; j < PER; ++j) f[j] = m[j];
        }
#pragma unroll
        for (int j = 0; j < PER; ++j)
#pragma unroll
          for (int e = 0; e < W; ++e) sum[e] = fmaf(f[j], v[j][e], sum[e]);
      } else if (in) {
        for (int j = 0; j < per; ++j) {
          float one[W];
          load_w<W>(base + j * p.D, one);
#pragma unroll
          for (int e = 0; e < W; ++e) sum[e] = fmaf(m[j], one[e], sum[e]);
        }
      }
      store_w<W>(out + ((size_t)h * p.G + c) * p.P + i, sum);
    }
  }
}

// NT threads a token: 256, or 1,024 for a few tokens whose product left split sums (a thread then walks one piece).
template <typename T, int NT, int W>
__global__ void __launch_bounds__(NT)
qkv_prepare_kernel(const Params p, T* __restrict__ pages, T* __restrict__ q_out) {
  tl::pdl_launch_dependents();
  extern __shared__ __align__(16) float smem[];
  __shared__ float scratch[32];
  const int t = blockIdx.x;
  const int qn = p.H * p.D, kn = p.G * p.D, vn = p.G * p.V, half = p.dims >> 1;
  float* mix = smem;                         // H H (rounded up to a multiple of 4)
  float* q = mix + p.mix_floats;             // H D
  float* k = q + qn;                         // G D
  float* v = k + kn;                         // G V
  float* cosines = v + (vn + 3) / 4 * 4;     // half
  float* sines = cosines + (half + 3) / 4 * 4;
  if (p.mix_floats && p.spread)  // weights: before the wait
    for (int i = threadIdx.x; i < p.H * p.H; i += NT) mix[i] = p.mix[i];
  tl::pdl_wait();
  const int pos = p.positions[t];
  const int req = p.token_req[t];
  const bool spread = p.mix && (p.spread == 1 || (p.spread == 2 && p.req_indptr[req + 1] - p.req_indptr[req] > 1));
  const float* row = p.src + (size_t)t * p.src_stride;
  float ssq = 0.f, ssk = 0.f;
  for (int i = threadIdx.x * W; i < qn + kn + vn; i += NT * W) {
    float x[W];
    if (p.splits == 1) {
      load_w<W>(row + i, x);
    } else {  // ascending splits, eight loads in flight
#pragma unroll
      for (int e = 0; e < W; ++e) x[e] = 0.f;
      for (int s = 0; s < p.splits; s += 8) {
        float one[8][W];
#pragma unroll
        for (int j = 0; j < 8; ++j)
          if (s + j < p.splits) load_w<W>(row + (size_t)(s + j) * p.split_stride + i, one[j]);
#pragma unroll
        for (int j = 0; j < 8; ++j)
          if (s + j < p.splits)
#pragma unroll
            for (int e = 0; e < W; ++e) x[e] += one[j][e];
      }
    }
    if (p.bias) {
      float b[W];
      load_w<W>(p.bias + i, b);
#pragma unroll
      for (int e = 0; e < W; ++e) x[e] += b[e];
    }
    store_w<W>(q + i, x);
#pragma unroll
    for (int e = 0; e < W; ++e) {
      if (i < qn) ssq = fmaf(x[e], x[e], ssq);
      else if (i < qn + kn) ssk = fmaf(x[e], x[e], ssk);
    }
  }
  for (int i = threadIdx.x; i < half; i += NT) {
    float sn, cs;
    sincosf((float)pos * p.inv_freq[i], &sn, &cs);
    cosines[i] = cs * p.magnitude;
    sines[i] = sn * p.magnitude;
  }
  const float inv_q = p.wq ? 1.f / sqrtf(block_sum<NT>(ssq, scratch) / (float)qn + p.eps) : 1.f;
  const float inv_k = p.wk ? 1.f / sqrtf(block_sum<NT>(ssk, scratch) / (float)kn + p.eps) : 1.f;
  __syncthreads();
  // norm and rotation, in place: the lower entries of rotated pairs do both
  const int turned = half / W, per_head = turned + (p.D - p.dims) / W;
  for (int item = threadIdx.x; item < (p.H + p.G) * per_head; item += NT) {
    const int head = item / per_head, i = item - head * per_head;
    const int e0 = i < turned ? i * W : i * W + half;
    float* x = q + (size_t)head * p.D + e0;
    const bool is_q = head < p.H;
    const float* w = is_q ? p.wq : p.wk;
    if (w) w += (size_t)(is_q ? head : head - p.H) * p.D + e0;
    const float inv = is_q ? inv_q : inv_k;
    float a[W], f[W];
    load_w<W>(x, a);
    if (w) {
      load_w<W>(w, f);
#pragma unroll
      for (int e = 0; e < W; ++e) a[e] = a[e] * inv * f[e];
    }
    if (i < turned) {
      float b[W], c[W], s[W], lo[W], hi[W];
      load_w<W>(x + half, b);
      if (w) {
        load_w<W>(w + half, f);
#pragma unroll
        for (int e = 0; e < W; ++e) b[e] = b[e] * inv * f[e];
      }
      load_w<W>(cosines + i * W, c);
      load_w<W>(sines + i * W, s);
#pragma unroll
      for (int e = 0; e < W; ++e) {
        lo[e] = a[e] * c[e] - b[e] * s[e];
        hi[e] = b[e] * c[e] + a[e] * s[e];
      }
      store_w<W>(x, lo);
      store_w<W>(x + half, hi);
    } else {
      store_w<W>(x, a);
    }
  }
  if (p.value_mode) {
    const float l = p.value_mode == 2 ? *p.lambda : 0.f;
    float* first = p.v_first + (size_t)t * vn;
    for (int i = threadIdx.x * W; i < vn; i += NT * W) {
      float mine[W], theirs[W];
      load_w<W>(v + i, mine);
      if (p.value_mode == 1) {
        store_w<W>(first + i, mine);
      } else {
        load_w<W>(first + i, theirs);
#pragma unroll
        for (int e = 0; e < W; ++e) mine[e] = (1.f - l) * mine[e] + l * theirs[e];
        store_w<W>(v + i, mine);
      }
    }
  }
  __syncthreads();
  const int pieces = p.P / W;
  // a row of n entries at ``src``, padded with zeros to P
  auto piece = [&](const float* src, int i, int n, float (&x)[W]) {
    if (i < n) {
      load_w<W>(src + i, x);
    } else {
#pragma unroll
      for (int e = 0; e < W; ++e) x[e] = 0.f;
    }
  };
  if (p.write_kv) {
    int page = -1;
    if (TL_DEBUG_OK(pos / p.page_size < p.table_width, TL_DEBUG_POSITION, pos))
      page = p.block_table[(size_t)req * p.table_width + pos / p.page_size];
    if (TL_DEBUG_OK(page >= 0 && page < p.num_pages, TL_DEBUG_PAGE, page) && page >= 0) {
      // pages: [num_pages, 2, G, page_size, P]
      T* dst = pages + (size_t)page * 2 * p.G * p.page_size * p.P + (size_t)(pos % p.page_size) * p.P;
      for (int item = threadIdx.x; item < 2 * p.G * pieces; item += NT) {
        const int head = item / pieces, i = (item - head * pieces) * W;  // key heads, then value heads
        const bool is_v = head >= p.G;
        float x[W];
        piece(is_v ? v + (size_t)(head - p.G) * p.V : k + (size_t)head * p.D, i, is_v ? p.V : p.D, x);
        store_w<W>(dst + (size_t)head * p.page_size * p.P + i, x);
      }
    }
  }
  T* out = q_out + (size_t)t * p.q_stride;
  if (!spread) {
    for (int item = threadIdx.x; item < p.H * pieces; item += NT) {
      const int head = item / pieces, i = (item - head * pieces) * W;
      float x[W];
      piece(q + (size_t)head * p.D, i, p.D, x);
      store_w<W>(out + (size_t)head * p.P + i, x);
    }
    return;
  }
  switch (p.H / p.G) {
    case 1: spread_queries<T, NT, 1, W>(p, q, mix, out); break;
    case 2: spread_queries<T, NT, 2, W>(p, q, mix, out); break;
    case 4: spread_queries<T, NT, 4, W>(p, q, mix, out); break;
    case 8: spread_queries<T, NT, 8, W>(p, q, mix, out); break;
    default: spread_queries<T, NT, 0, W>(p, q, mix, out); break;
  }
}

template <typename T, int NT, int W>
int launch(const Params& p, void* pages, void* q_out, int tokens, size_t smem, cudaStream_t stream) {
  if (smem > 48 * 1024) {
    const cudaError_t err = cudaFuncSetAttribute(qkv_prepare_kernel<T, NT, W>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
  }
  tl::launch_kernel(qkv_prepare_kernel<T, NT, W>, (unsigned)tokens, NT, smem, stream, p, (T*)pages, (T*)q_out);
  return TL_LAUNCH_CHECK();
}

template <typename T>
int pick(Params p, void* pages, void* q_out, int tokens, cudaStream_t stream) {
  p.mix_floats = p.mix ? (p.H * p.H + 3) / 4 * 4 : 0;
  const size_t half = p.dims / 2, vn = (size_t)p.G * p.V;
  const size_t floats = p.mix_floats + (size_t)(p.H + p.G) * p.D + (vn + 3) / 4 * 4 + 2 * ((half + 3) / 4 * 4);
  const size_t smem = floats * sizeof(float);
  if (smem > 200 * 1024) return TL_ERR_UNSUPPORTED;
  uintptr_t all = 0;
  for (const void* x : {(const void*)p.src, (const void*)p.bias, (const void*)p.wq, (const void*)p.wk, (const void*)p.v_first,
                        (const void*)pages, (const void*)q_out})
    all |= reinterpret_cast<uintptr_t>(x);
  // 16-byte pieces; the choice of kernel depends on sizes and alignment (and on split sums) alone, never on the batch
  const bool wide = p.D % 4 == 0 && p.V % 4 == 0 && p.dims % 8 == 0 && p.P % 4 == 0 && p.src_stride % 4 == 0 &&
                    p.split_stride % 4 == 0 && p.q_stride % 4 == 0 && (all & 15) == 0;
  if (p.splits > 1)
    return wide ? launch<T, 1024, 4>(p, pages, q_out, tokens, smem, stream) : launch<T, 1024, 1>(p, pages, q_out, tokens, smem, stream);
  return wide ? launch<T, 256, 4>(p, pages, q_out, tokens, smem, stream) : launch<T, 256, 1>(p, pages, q_out, tokens, smem, stream);
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
  return dtype == TL_DTYPE_F32 ? pick<float>(p, pages, q_out, tokens, stream)
                               : pick<__nv_bfloat16>(p, pages, q_out, tokens, stream);
}
