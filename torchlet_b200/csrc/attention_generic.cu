// Paged causal grouped-query attention for any batch of (request, next tokens):
// prompt portions with cached context before them and single decoded tokens alike.
// One warp per (token, query head); keys are visited in tiles of 32 consecutive
// ABSOLUTE positions (tile edges at multiples of 32), so the order of every sum
// depends only on the token's position and window, never on how the sequence was cut
// into steps, on the batch, or on the pages used.  Scores, softmax and the weighted
// sum are float32; T is the storage type of queries, pages and output.
//
// Options: ``softcap`` > 0 bounds a score, s <- softcap tanh(s / softcap); ``sink`` adds one to the
// softmax's denominator (a key of score 0 that has no value), or with ``sink_values`` exp(sink_values[head]); ``gate`` (float32 rows) multiplies the
// output element by element with sigmoid(gate).
//
// ``keep`` > 0: the first ``keep`` positions of the sequence are visible beside the window (their tiles come first).
// ``chunks`` = nkv: a query row spans the keys of ALL KV heads, [nh][nkv][d], and a head's score is the sum over them
// (scores mixed across the heads, folded into the queries; see csrc/qkv_prepare.cu); 1: the head's own KV head alone.
// ``v_cols``: how many entries of a value row are written for a head (the cache rows may be padded).
//
// This is the true 32-bit kernel and the any-size bfloat16 kernel (head_dim up to 256: keys are
// read eight entries at a time where head_dim and the query stride are multiples of 8, one at a
// time otherwise; any head counts, any page size).
//
// Reference counterparts: forward_ragged_attention_kernel and
// forward_slot_attention_decode_kernel, v10_triton_paged_gqa/kernel/gqa.py:5-228
// (query head h reads KV head h // g, scale head_dim^-0.5, key allowed iff
// key_pos <= query_pos, online softmax, acc / l).
#include <math.h>

#include "common.cuh"

namespace {

using namespace tl;

constexpr int WARPS = 4;
constexpr int MAX_D = 256;

template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
attention_generic_kernel(const T* __restrict__ q, int q_stride, const T* __restrict__ pages,
                         const int* __restrict__ block_table, int table_width,
                         const int* __restrict__ token_req, const int* __restrict__ positions,
                         T* __restrict__ out, int out_stride, int tokens, int nh, int nkv, int d,
                         int page_size, int window, float scale, int num_pages, float softcap, int sink,
                         const float* __restrict__ sink_values, const float* __restrict__ gate, int gate_stride, int wide,
                         int keep, int chunks, int v_cols) {
  tl::pdl_wait();               // everything before us in the stream is complete and visible
  tl::pdl_launch_dependents();  // the next kernel may start its own prologue

  extern __shared__ __align__(16) float all_queries[];  // [WARPS][chunks d]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * WARPS + warp;
  if (item >= (long long)tokens * nh) return;
  const int t = (int)(item / nh), h = (int)(item % nh);
  const int kvh = h / (nh / nkv);
  const int pos = positions[t];
  const int lo = first_key(pos, window);
  const int* table = block_table + (size_t)token_req[t] * table_width;

  const int q_len = chunks * d;
  float* qs = all_queries + warp * q_len;
  const T* qrow = q + (size_t)t * q_stride + (size_t)h * q_len;
  for (int i = lane; i < q_len; i += 32) qs[i] = to_float(qrow[i]);
  __syncwarp();

  const size_t page_elems = (size_t)2 * nkv * page_size * d;
  const size_t k_off = chunks > 1 ? 0 : (size_t)kvh * page_size * d;
  const size_t head_step = (size_t)page_size * d;  // from a key to the next KV head's
  const size_t v_off = ((size_t)nkv + kvh) * page_size * d;

  // the sink is a key of a given score (0, or the head's own number) and no value that every query sees: the running
  // maximum starts at that score with a weight of exp(0) in the denominator
  float m = sink ? (sink_values ? sink_values[h] : 0.f) : -INFINITY, l = sink ? 1.f : 0.f;
  float acc[MAX_D / 32];
#pragma unroll
  for (int c = 0; c < MAX_D / 32; ++c) acc[c] = 0.f;

  // tiles of kept first positions that lie wholly before the window's first tile, then the window's
  const int window_start = lo & ~31;
  const int kept_end = keep < window_start ? (keep + 31) & ~31 : window_start;
  for (int start = kept_end > 0 ? 0 : window_start; start <= pos;
       start = start + 32 == kept_end ? window_start : start + 32) {
    const int key = start + lane;
    const bool valid = (key >= lo || key < keep) && key <= pos;
    float s = -INFINITY;
    size_t row_off = 0;
    if (valid) {
      int page = 0;  // a key whose table entry fails a debug-build check is read from the reserved page 0
      if (TL_DEBUG_OK(key / page_size < table_width, TL_DEBUG_POSITION, key)) page = table[key / page_size];
      if (!TL_DEBUG_OK(page >= 0 && page < num_pages, TL_DEBUG_PAGE, page)) page = 0;
      row_off = (size_t)page * page_elems + (size_t)(key % page_size) * d;
      const T* krow = pages + row_off + k_off;
      float dot = 0.f;
      for (int c = 0; c < chunks; ++c, krow += head_step) {
        const float* qc = qs + c * d;
        if (wide) {
          for (int i = 0; i < d; i += 8) {
            float kv[8];
            load8(krow + i, kv);
#pragma unroll
            for (int j = 0; j < 8; ++j) dot = fmaf(qc[i + j], kv[j], dot);
          }
        } else {  // the same order of additions, one entry at a time
          for (int i = 0; i < d; ++i) dot = fmaf(qc[i], to_float(krow[i]), dot);
        }
      }
      s = dot * scale;
      if (softcap > 0.f) s = softcap * tanhf(s / softcap);
    }
    const float new_m = fmaxf(m, warp_max(s));
    const float corr = expf(m - new_m);  // first tile: exp(-inf) = 0
    const float p = valid ? expf(s - new_m) : 0.f;
    l = l * corr + warp_sum(p);
    m = new_m;
#pragma unroll
    for (int c = 0; c < MAX_D / 32; ++c) acc[c] *= corr;
    const int first = start >= keep && lo > start ? lo - start : 0;  // (a lane without a key has weight 0 and is skipped)
    const int last = pos - start < 31 ? pos - start : 31;
    for (int j = first; j <= last; ++j) {
      if (keep && !__shfl_sync(0xffffffffu, (int)valid, j)) continue;
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const size_t off = __shfl_sync(0xffffffffu, (unsigned long long)row_off, j);
      const T* vrow = pages + off + v_off;
#pragma unroll
      for (int c = 0; c < MAX_D / 32; ++c) {
        const int i = lane + 32 * c;
        if (i < d) acc[c] = fmaf(pj, to_float(vrow[i]), acc[c]);
      }
    }
  }
  T* orow = out + (size_t)t * out_stride + (size_t)h * v_cols;
  const float inv = 1.f / l;
#pragma unroll
  for (int c = 0; c < MAX_D / 32; ++c) {
    const int i = lane + 32 * c;
    if (i < v_cols) {
      float v = acc[c] * inv;
      if (gate) v *= 1.f / (1.f + expf(-gate[(size_t)t * gate_stride + (size_t)h * d + i]));
      orow[i] = from_float<T>(v);
    }
  }
}

}  // namespace

TL_DEBUG_READER(tl_attention_generic_debug_error)

extern "C" int tl_attention_generic(const void* q, int q_stride, const void* pages, int dtype,
                                    const int* block_table, int table_width, const int* token_req,
                                    const int* positions, void* out, int out_stride, int tokens,
                                    int nh, int nkv, int d, int page_size, int window, float scale,
                                    int num_pages, float softcap, int sink, const float* sink_values,
                                    const float* gate, int gate_stride, int keep, int chunks, int v_cols,
                                    cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (d <= 0 || d > MAX_D || nkv <= 0 || nh % nkv || page_size <= 0) return TL_ERR_UNSUPPORTED;
  if (keep < 0 || (chunks != 1 && chunks != nkv) || v_cols <= 0 || v_cols > d) return TL_ERR_UNSUPPORTED;
  const size_t smem = (size_t)WARPS * chunks * d * sizeof(float);
  if (smem > 200 * 1024) return TL_ERR_UNSUPPORTED;
  if (smem > 48 * 1024) {
    const cudaError_t err = dtype == TL_DTYPE_F32
        ? cudaFuncSetAttribute(attention_generic_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)
        : cudaFuncSetAttribute(attention_generic_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
  }
  const int wide = d % 8 == 0 && q_stride % 8 == 0 && (reinterpret_cast<uintptr_t>(pages) & 31) == 0;
  const long long items = (long long)tokens * nh;
  const unsigned blocks = (unsigned)((items + WARPS - 1) / WARPS);
  if (dtype == TL_DTYPE_F32)
    tl::launch_kernel(attention_generic_kernel<float>, blocks, WARPS * 32, smem, stream,
        (const float*)q, q_stride, (const float*)pages, block_table, table_width, token_req,
        positions, (float*)out, out_stride, tokens, nh, nkv, d, page_size, window, scale, num_pages, softcap, sink,
        sink_values, gate, gate_stride, wide, keep, chunks, v_cols);
  else
    tl::launch_kernel(attention_generic_kernel<__nv_bfloat16>, blocks, WARPS * 32, smem, stream,
        (const __nv_bfloat16*)q, q_stride, (const __nv_bfloat16*)pages, block_table, table_width,
        token_req, positions, (__nv_bfloat16*)out, out_stride, tokens, nh, nkv, d, page_size, window,
        scale, num_pages, softcap, sink, sink_values, gate, gate_stride, wide, keep, chunks, v_cols);
  return TL_LAUNCH_CHECK();
}
