// What stands between the input product and the attention kernel of a mixer whose queries and keys
// are normed over the WHOLE projection and whose values may be the keys themselves.  One block per
// token; the projections arrive as float32 rows
//   proj[t] = [ q (H D) | k (G D) | ... ]
// (with separate values: [ q | k | v (G D) | ... ]).  In float32:
//   q <- q / rms(q over all H D) * wq,   k' <- k / rms(k over all G D) * wk      (plain weights);
//   the first ``dims`` entries of every head of q and k' are rotated by the token's position, entry i
//   paired with i + dims / 2: (u, v) -> (u c - v s, v c + u s), c = m cos(p f_i), s = m sin(p f_i), with
//   the frequencies f (``inv_freq``, dims / 2 floats) and the magnitude m given by the host;
//   q goes to ``q_out`` in the compute type, k' to plane 0 of the token's cache row and the value to
//   plane 1: the key AS PROJECTED (before norm and rotation) where the values are the keys.  Values may turn by
//   position as well (``v_inv_freq``: entry i of a value head with i + v_half, i < v_half; no magnitude).
// The cosines and sines of a token are taken once for all heads.
//
// head_finish is what stands BEHIND the attention kernel of such a mixer: rotated values leave a head's output turned,
// so it is turned back by the token's own position (the same pairs, the opposite angle), and a gate of one number a
// head multiplies it, out[t, h] = turn_back(o[t, h]) * sigmoid(gate[t, h]), in place.
#include <math.h>

#include "common.cuh"

namespace {

using namespace tl;

constexpr int MAX_HALF = 128;  // rotated pairs of a head of up to 256 entries

template <int V> __device__ __forceinline__ void load_some(const float* p, float (&v)[V]) {
#pragma unroll
  for (int j = 0; j < V; j += 4) {
    if constexpr (V % 4 == 0) {
      const float4 x = *reinterpret_cast<const float4*>(p + j);
      v[j] = x.x; v[j + 1] = x.y; v[j + 2] = x.z; v[j + 3] = x.w;
    } else {
      v[j] = p[j];
    }
  }
}
template <int V> __device__ __forceinline__ void load_some(const __nv_bfloat16* p, float (&v)[V]) {
  if constexpr (V == 8) load8(p, v);
  else v[0] = __bfloat162float(*p);
}
template <int V> __device__ __forceinline__ void store_some(float* p, const float (&v)[V]) {
#pragma unroll
  for (int j = 0; j < V; j += 4) {
    if constexpr (V % 4 == 0) *reinterpret_cast<float4*>(p + j) = make_float4(v[j], v[j + 1], v[j + 2], v[j + 3]);
    else p[j] = v[j];
  }
}
template <int V> __device__ __forceinline__ void store_some(__nv_bfloat16* p, const float (&v)[V]) {
  if constexpr (V == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
  } else if constexpr (V == 8) {
    uint32_t w[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
      w[j] = *reinterpret_cast<const uint32_t*>(&h);
    }
    *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  } else {
    *p = __float2bfloat16_rn(v[0]);
  }
}

// NT threads a token: 256 up to 1,024 entries of q and k together, 512 up to 4,096, 1,024 beyond, so that a thread
// walks few entries one after the other.
template <typename T, int NT>
__global__ void __launch_bounds__(NT)
normed_qk_store_kernel(const float* __restrict__ proj, int proj_stride, const float* __restrict__ wq,
                       const float* __restrict__ wk, const float* __restrict__ inv_freq, float magnitude, float eps,
                       const int* __restrict__ positions, const int* __restrict__ token_req,
                       const int* __restrict__ block_table, int table_width, T* __restrict__ pages, int page_size,
                       int num_pages, T* __restrict__ q_out, int nh, int nkv, int d, int dims, int norm_q, int norm_k,
                       int v_offset, int write_kv, const float* __restrict__ v_inv_freq, int v_half) {
  tl::pdl_launch_dependents();
  tl::pdl_wait();
  __shared__ float scratch[32];
  __shared__ float turn[4][MAX_HALF];  // cos and sin of the keys' angles (times the magnitude), of the values'
  const int t = blockIdx.x;
  const float* row = proj + (size_t)t * proj_stride;
  const int qn = nh * d, kn = nkv * d, half = dims >> 1;
  const int pos = positions[t];
  const float p = (float)pos;
  for (int i = threadIdx.x; i < half + v_half; i += NT) {
    float sn, cs;
    if (i < half) {
      sincosf(p * inv_freq[i], &sn, &cs);
      turn[0][i] = cs * magnitude;
      turn[1][i] = sn * magnitude;
    } else {
      sincosf(p * v_inv_freq[i - half], &sn, &cs);
      turn[2][i - half] = cs;
      turn[3][i - half] = sn;
    }
  }
  float ssq = 0.f, ssk = 0.f;
  if (norm_q)
    for (int i = threadIdx.x; i < qn; i += NT) ssq = fmaf(row[i], row[i], ssq);
  if (norm_k)
    for (int i = threadIdx.x; i < kn; i += NT) ssk = fmaf(row[qn + i], row[qn + i], ssk);
  if (norm_q) ssq = block_sum<NT>(ssq, scratch);
  if (norm_k) ssk = block_sum<NT>(ssk, scratch);
  __syncthreads();
  const float inv_q = norm_q ? 1.f / sqrtf(ssq / (float)qn + eps) : 1.f;
  const float inv_k = norm_k ? 1.f / sqrtf(ssk / (float)kn + eps) : 1.f;

  // queries: entry e of head h; the lower entry of a rotated pair does both
  for (int c = threadIdx.x; c < qn; c += NT) {
    const int e = c % d;
    if (e >= half && e < dims) continue;
    const float a = row[c] * inv_q * (norm_q ? wq[c] : 1.f);
    if (e < half) {
      const float b = row[c + half] * inv_q * (norm_q ? wq[c + half] : 1.f);
      const float cs = turn[0][e], sn = turn[1][e];
      q_out[(size_t)t * qn + c] = from_float<T>(a * cs - b * sn);
      q_out[(size_t)t * qn + c + half] = from_float<T>(b * cs + a * sn);
    } else {
      q_out[(size_t)t * qn + c] = from_float<T>(a);
    }
  }
  if (!write_kv) return;
  int page = 0;
  if (TL_DEBUG_OK(pos / page_size < table_width, TL_DEBUG_POSITION, pos))
    page = block_table[(size_t)token_req[t] * table_width + pos / page_size];
  if (!TL_DEBUG_OK(page >= 0 && page < num_pages, TL_DEBUG_PAGE, page)) return;
  // pages: [num_pages, 2, nkv, page_size, d]
  T* kdst = pages + (size_t)page * 2 * nkv * page_size * d + (size_t)(pos % page_size) * d;
  T* vdst = kdst + (size_t)nkv * page_size * d;
  for (int c = threadIdx.x; c < kn; c += NT) {
    const int g = c / d, e = c - g * d;
    const size_t at = (size_t)g * page_size * d + e;
    if (e < v_half) {
      const float a = row[v_offset + c], b = row[v_offset + c + v_half];
      const float cs = turn[2][e], sn = turn[3][e];
      vdst[at] = from_float<T>(a * cs - b * sn);
      vdst[at + v_half] = from_float<T>(b * cs + a * sn);
    } else if (e >= 2 * v_half) {
      vdst[at] = from_float<T>(row[v_offset + c]);
    }
    if (e >= half && e < dims) continue;
    const float a = row[qn + c] * inv_k * (norm_k ? wk[c] : 1.f);
    if (e < half) {
      const float b = row[qn + c + half] * inv_k * (norm_k ? wk[c + half] : 1.f);
      const float cs = turn[0][e], sn = turn[1][e];
      kdst[at] = from_float<T>(a * cs - b * sn);
      kdst[at + half] = from_float<T>(b * cs + a * sn);
    } else {
      kdst[at] = from_float<T>(a);
    }
  }
}

// The same where every size is a multiple of 4 and everything is 16-byte aligned: a thread takes four neighbouring pairs (or
// four entries that do not turn) of a head at a time, and has its first ones on their way before the cosines are taken.
template <typename T, int NT>
__global__ void __launch_bounds__(NT)
normed_qk_store_wide_kernel(const float* __restrict__ proj, int proj_stride, const float* __restrict__ wq,
                            const float* __restrict__ wk, const float* __restrict__ inv_freq, float magnitude, float eps,
                            const int* __restrict__ positions, const int* __restrict__ token_req,
                            const int* __restrict__ block_table, int table_width, T* __restrict__ pages, int page_size,
                            int num_pages, T* __restrict__ q_out, int nh, int nkv, int d, int dims, int norm_q, int norm_k,
                            int v_offset, int write_kv, const float* __restrict__ v_inv_freq, int v_half) {
  tl::pdl_launch_dependents();
  tl::pdl_wait();
  __shared__ float scratch[32];
  __shared__ __align__(16) float turn[4][MAX_HALF];
  const int t = blockIdx.x;
  const float* row = proj + (size_t)t * proj_stride;
  const int qn = nh * d, kn = nkv * d, half = dims >> 1;
  const int pos = positions[t];
  const float p = (float)pos;
  // items: the quads of the q heads, then of the k heads, then of the v heads
  const int per_qk = (half >> 2) + ((d - dims) >> 2), per_v = (v_half >> 2) + ((d - 2 * v_half) >> 2);
  const int q_items = nh * per_qk, k_items = write_kv ? nkv * per_qk : 0, v_items = write_kv ? nkv * per_v : 0;
  const int items = q_items + k_items + v_items;
  struct Quad {
    int what, head, e, partner;  // 0 q, 1 k, 2 v; the entry in its head; how far the partner stands (0: it does not turn)
  };
  auto quad_of = [&](int item) {
    Quad x;
    x.what = item < q_items ? 0 : (item < q_items + k_items ? 1 : 2);
    const int local = x.what == 0 ? item : (x.what == 1 ? item - q_items : item - q_items - k_items);
    const int per = x.what == 2 ? per_v : per_qk, n = x.what == 2 ? v_half : half;
    x.head = local / per;
    const int i = local - x.head * per;
    x.partner = i < (n >> 2) ? n : 0;
    x.e = x.partner ? i * 4 : 2 * n + (i - (n >> 2)) * 4;
    return x;
  };
  auto source = [&](const Quad& x) { return row + (x.what == 0 ? 0 : (x.what == 1 ? qn : v_offset)) + x.head * d + x.e; };
  float a[4], b[4];
  auto fetch = [&](const Quad& x) {
    const float* src = source(x);
    load_some<4>(src, a);
    if (x.partner) load_some<4>(src + x.partner, b);
  };
  Quad now{};
  if (threadIdx.x < items) {
    now = quad_of(threadIdx.x);
    fetch(now);
  }
  for (int i = threadIdx.x; i < half + v_half; i += NT) {
    float sn, cs;
    if (i < half) {
      sincosf(p * inv_freq[i], &sn, &cs);
      turn[0][i] = cs * magnitude;
      turn[1][i] = sn * magnitude;
    } else {
      sincosf(p * v_inv_freq[i - half], &sn, &cs);
      turn[2][i - half] = cs;
      turn[3][i - half] = sn;
    }
  }
  float inv_q = 1.f, inv_k = 1.f;
  auto mean_square = [&](const float* x, int n) {
    float ss = 0.f;
    for (int i = threadIdx.x * 4; i < n; i += NT * 4) {
      const float4 v = *reinterpret_cast<const float4*>(x + i);
      ss = fmaf(v.x, v.x, ss);
      ss = fmaf(v.y, v.y, ss);
      ss = fmaf(v.z, v.z, ss);
      ss = fmaf(v.w, v.w, ss);
    }
    return block_sum<NT>(ss, scratch) / (float)n;
  };
  if (norm_q) inv_q = 1.f / sqrtf(mean_square(row, qn) + eps);
  if (norm_k) inv_k = 1.f / sqrtf(mean_square(row + qn, kn) + eps);
  __syncthreads();
  // pages: [num_pages, 2, nkv, page_size, d]
  T* kdst = nullptr;
  if (write_kv) {
    int page = -1;
    if (TL_DEBUG_OK(pos / page_size < table_width, TL_DEBUG_POSITION, pos))
      page = block_table[(size_t)token_req[t] * table_width + pos / page_size];
    if (TL_DEBUG_OK(page >= 0 && page < num_pages, TL_DEBUG_PAGE, page) && page >= 0)
      kdst = pages + (size_t)page * 2 * nkv * page_size * d + (size_t)(pos % page_size) * d;
  }
  for (int item = threadIdx.x; item < items;) {
    const float inv = now.what == 0 ? inv_q : (now.what == 1 ? inv_k : 1.f);
    const float* w = now.what == 0 ? (norm_q ? wq : nullptr) : (now.what == 1 && norm_k ? wk : nullptr);
    const int at = now.head * d + now.e;
    float x[4], y[4];
    if (w) {
      float wa[4];
      load_some<4>(w + at, wa);
#pragma unroll
      for (int j = 0; j < 4; ++j) a[j] = a[j] * inv * wa[j];
      if (now.partner) {
        load_some<4>(w + at + now.partner, wa);
#pragma unroll
        for (int j = 0; j < 4; ++j) b[j] = b[j] * inv * wa[j];
      }
    }
    if (now.partner) {
      float cs[4], sn[4];
      load_some<4>(&turn[now.what == 2 ? 2 : 0][now.e], cs);
      load_some<4>(&turn[now.what == 2 ? 3 : 1][now.e], sn);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        x[j] = a[j] * cs[j] - b[j] * sn[j];
        y[j] = b[j] * cs[j] + a[j] * sn[j];
      }
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j) x[j] = a[j];
    }
    T* dst = q_out + (size_t)t * qn + at;
    if (now.what != 0)
      dst = kdst ? kdst + (size_t)((now.what == 2 ? nkv : 0) + now.head) * page_size * d + now.e : nullptr;
    const int partner = now.partner;
    item += NT;
    if (item < items) {
      now = quad_of(item);
      fetch(now);
    }
    if (dst) {
      store_some<4>(dst, x);
      if (partner) store_some<4>(dst + partner, y);
    }
  }
}

// One block a token; a thread takes V neighbouring pairs of a head at a time (V = 8 where the sizes allow, else 1).
// rows [tokens][nh][d]: entries past 2 v_half of a head only take the gate.
template <typename T, int V>
__global__ void __launch_bounds__(128)
head_finish_kernel(T* __restrict__ rows, const int* __restrict__ positions, const float* __restrict__ v_inv_freq,
                   const float* __restrict__ gate, int gate_stride, int nh, int d, int v_half) {
  tl::pdl_launch_dependents();
  __shared__ float cosines[MAX_HALF], sines[MAX_HALF];
  const int t = blockIdx.x;
  const float p = (float)positions[t];  // written before the step's first kernel or by the step's gather, which none overlaps
  for (int i = threadIdx.x; i < v_half; i += 128) sincosf(p * v_inv_freq[i], &sines[i], &cosines[i]);
  tl::pdl_wait();
  __syncthreads();
  T* row = rows + (size_t)t * nh * d;
  const int per_head = v_half / V + (d - 2 * v_half);
  for (int e = threadIdx.x; e < nh * per_head; e += 128) {
    const int h = e / per_head, i = e - h * per_head;
    const float g = gate ? 1.f / (1.f + expf(-gate[(size_t)t * gate_stride + h])) : 1.f;
    T* head = row + (size_t)h * d;
    if (i < v_half / V) {
      float a[V], b[V], u[V], w[V];
      load_some<V>(head + i * V, a);
      load_some<V>(head + i * V + v_half, b);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        const float cs = cosines[i * V + j], sn = sines[i * V + j];
        u[j] = (a[j] * cs + b[j] * sn) * g;
        w[j] = (b[j] * cs - a[j] * sn) * g;
      }
      store_some<V>(head + i * V, u);
      store_some<V>(head + i * V + v_half, w);
    } else {
      T* at = head + 2 * v_half + (i - v_half / V);
      *at = from_float<T>(to_float(*at) * g);
    }
  }
}

}  // namespace

TL_DEBUG_READER(tl_gated_attention_debug_error)

// rows [tokens][nh d] (the compute type), in place; v_half 0: no rotation; gate (float32 rows of one number a head,
// or null: no gate).
extern "C" int tl_head_finish(void* rows, int dtype, const int* positions, const float* v_inv_freq, const float* gate,
                              int gate_stride, int tokens, int nh, int d, int v_half, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (nh <= 0 || d <= 0 || v_half < 0 || 2 * v_half > d || v_half > MAX_HALF || (v_half && !v_inv_freq)) return TL_ERR_UNSUPPORTED;
  const bool wide = v_half % 8 == 0 && d % 8 == 0 && (reinterpret_cast<uintptr_t>(rows) & 15) == 0;
#define TL_FINISH(T, V)                                                                                             \
  tl::launch_kernel(head_finish_kernel<T, V>, (unsigned)tokens, 128, 0, stream, (T*)rows, positions, v_inv_freq, gate, \
                    gate_stride, nh, d, v_half)
  if (dtype == TL_DTYPE_F32) {
    if (wide) TL_FINISH(float, 8);
    else TL_FINISH(float, 1);
  } else {
    if (wide) TL_FINISH(__nv_bfloat16, 8);
    else TL_FINISH(__nv_bfloat16, 1);
  }
#undef TL_FINISH
  return TL_LAUNCH_CHECK();
}

extern "C" int tl_normed_qk_store(const float* proj, int proj_stride, const float* wq, const float* wk,
                                  const float* inv_freq, float magnitude, float eps, const int* positions,
                                  const int* token_req, const int* block_table, int table_width, void* pages, int dtype,
                                  int page_size, int num_pages, void* q_out, int tokens, int nh, int nkv, int d, int dims,
                                  int norm_q, int norm_k, int v_offset, int write_kv, const float* v_inv_freq,
                                  int v_half, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (d <= 0 || dims < 0 || dims > d || dims % 2 || nh <= 0 || nkv <= 0 || page_size <= 0) return TL_ERR_UNSUPPORTED;
  if (dims / 2 > MAX_HALF || v_half < 0 || v_half > MAX_HALF || 2 * v_half > d || (v_half && !v_inv_freq)) return TL_ERR_UNSUPPORTED;
  const long long width = (long long)(nh + nkv) * d;
  const uintptr_t all = (uintptr_t)proj | (uintptr_t)wq | (uintptr_t)wk | (uintptr_t)pages | (uintptr_t)q_out;
  if (d % 4 == 0 && dims % 8 == 0 && v_half % 4 == 0 && proj_stride % 4 == 0 && v_offset % 4 == 0 && (all & 15) == 0) {
#define TL_STORE_WIDE(T, NT)                                                                                               \
  tl::launch_kernel(normed_qk_store_wide_kernel<T, NT>, (unsigned)tokens, NT, 0, stream, proj, proj_stride, wq, wk, inv_freq, \
                    magnitude, eps, positions, token_req, block_table, table_width, (T*)pages, page_size, num_pages,         \
                    (T*)q_out, nh, nkv, d, dims, norm_q, norm_k, v_offset, write_kv, v_inv_freq, v_half)
    if (dtype == TL_DTYPE_F32) {
      if (width <= 2048) TL_STORE_WIDE(float, 128);
      else TL_STORE_WIDE(float, 256);
    } else {
      if (width <= 2048) TL_STORE_WIDE(__nv_bfloat16, 128);
      else TL_STORE_WIDE(__nv_bfloat16, 256);
    }
#undef TL_STORE_WIDE
    return TL_LAUNCH_CHECK();
  }
#define TL_STORE(T, NT)                                                                                              \
  tl::launch_kernel(normed_qk_store_kernel<T, NT>, (unsigned)tokens, NT, 0, stream, proj, proj_stride, wq, wk, inv_freq, \
                    magnitude, eps, positions, token_req, block_table, table_width, (T*)pages, page_size, num_pages,     \
                    (T*)q_out, nh, nkv, d, dims, norm_q, norm_k, v_offset, write_kv,        \
                    v_inv_freq, v_half)
  if (dtype == TL_DTYPE_F32) {
    if (width <= 1024) TL_STORE(float, 256);
    else if (width <= 4096) TL_STORE(float, 512);
    else TL_STORE(float, 1024);
  } else {
    if (width <= 1024) TL_STORE(__nv_bfloat16, 256);
    else if (width <= 4096) TL_STORE(__nv_bfloat16, 512);
    else TL_STORE(__nv_bfloat16, 1024);
  }
#undef TL_STORE
  return TL_LAUNCH_CHECK();
}
