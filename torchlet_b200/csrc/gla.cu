// Gated linear attention: a recurrent mixer whose per-request state is one D x V float32 matrix
// per head (key channel i, value channel j), carried from token to token:
//
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T,      o_t = S_t^T q_t * qscale
//
// with a decay per key channel a = sigmoid(z)^(1/tau) = exp(logsigmoid(z) / tau), z = W2 l + b, where
// l is a low-rank projection of the layer's input.  Everything here is float32, also in the bfloat16
// engine: the projections arrive as float32 rows
//   proj[t] = [ q (H D) | k (H D) | v (H V) | g (H V) | l (rank) ],
// or with q, k and v in planes of their own (the scan takes the distances from q to k and to v).
//
// A time-mixing recurrence with a bonus for the current token is the same scan with one more vector u per head:
//   o_t = (S_(t-1) + diag(u) k_t v_t^T)^T q_t,      S_t = diag(a_t) S_(t-1) + k_t v_t^T,
// whose decay is a = exp(-exp(z)), z = W2 tanh(l) + b.
//
// Three kernels:
//   decay   one block per (8 tokens, 128 or 512 channels): a of every key channel;
//   scan    one block per (request, head, 32 value channels): the columns of S are independent of one
//           another; four lanes share a column, each keeps a quarter of it in registers, and the block
//           walks the request's tokens of this step in order; q, k, a, v of a few tokens at a time are
//           staged in shared memory (four stages, asynchronous copies).  The state row of the request's slot
//           is read at the start and written back at the end, so a prompt cut into portions, or
//           decoded token by token, runs the same additions in the same order as the whole prompt;
//   finish  one warp per (token, head): o / rms(o) * weight * silu(g) in the compute type (the
//           weight covers one head and is shared by all, or has every head's own numbers).
#include <math.h>

#include "common.cuh"

namespace {

using namespace tl;

constexpr int DECAY_TOKENS = 8;
constexpr int DECAY_NT = 128;

// w2t: W2 transposed, [rank, channels]; out: [tokens, channels].  TANH: exp(-exp(z)) of a tanh of the low-rank input, else
// sigmoid(z)^(inv_tau).  A thread takes CH neighbouring channels: four where the grid is large anyway (a shared-memory read
// of the low-rank input then serves four channels, and those reads are what a long prompt's time goes into), one otherwise.
template <bool TANH, int CH>
__global__ void __launch_bounds__(DECAY_NT)
gla_decay_kernel(const float* __restrict__ proj, int proj_stride, int low_offset, const float* __restrict__ w2t,
                 const float* __restrict__ bias, float* __restrict__ out, int tokens, int channels, int rank,
                 float inv_tau) {
  tl::pdl_launch_dependents();
  tl::pdl_wait();
  extern __shared__ __align__(16) float low[];  // DECAY_TOKENS x the rank rounded up to a multiple of 4
  const int stride = (rank + 3) & ~3;
  const int t0 = blockIdx.x * DECAY_TOKENS;
  const int count = tokens - t0 < DECAY_TOKENS ? tokens - t0 : DECAY_TOKENS;
  for (int e = threadIdx.x; e < DECAY_TOKENS * stride; e += DECAY_NT) {
    const int tt = e / stride, j = e - tt * stride;
    const float l = tt < count && j < rank ? proj[(size_t)(t0 + tt) * proj_stride + low_offset + j] : 0.f;
    low[e] = TANH ? tanhf(l) : l;
  }
  __syncthreads();
  const int c = (blockIdx.y * DECAY_NT + threadIdx.x) * CH;
  if (c >= channels) return;
  float z[DECAY_TOKENS][CH];
#pragma unroll
  for (int tt = 0; tt < DECAY_TOKENS; ++tt)
#pragma unroll
    for (int k = 0; k < CH; ++k) z[tt][k] = 0.f;
#pragma unroll(CH == 1 ? 4 : 1)
  for (int j = 0; j < rank; j += 4) {  // ascending j: the order depends on the rank alone
    float w[4][CH];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float* src = w2t + (size_t)(j + i) * channels + c;
      if constexpr (CH == 4) {
        const float4 v = j + i < rank ? *reinterpret_cast<const float4*>(src) : make_float4(0.f, 0.f, 0.f, 0.f);
        w[i][0] = v.x; w[i][1] = v.y; w[i][2] = v.z; w[i][3] = v.w;
      } else {
        w[i][0] = j + i < rank ? *src : 0.f;
      }
    }
#pragma unroll
    for (int tt = 0; tt < DECAY_TOKENS; ++tt) {
      const float4 l = *reinterpret_cast<const float4*>(low + tt * stride + j);
#pragma unroll
      for (int k = 0; k < CH; ++k) {
        z[tt][k] = fmaf(w[0][k], l.x, z[tt][k]);
        z[tt][k] = fmaf(w[1][k], l.y, z[tt][k]);
        z[tt][k] = fmaf(w[2][k], l.z, z[tt][k]);
        z[tt][k] = fmaf(w[3][k], l.w, z[tt][k]);
      }
    }
  }
  float b[CH];
#pragma unroll
  for (int k = 0; k < CH; ++k) b[k] = bias[c + k];
#pragma unroll
  for (int tt = 0; tt < DECAY_TOKENS; ++tt) {
    if (tt >= count) break;
    float a[CH];
#pragma unroll
    for (int k = 0; k < CH; ++k) {
      const float x = z[tt][k] + b[k];
      if constexpr (TANH) {
        a[k] = expf(-expf(x));
      } else {
        // log(sigmoid(x)) = min(x, 0) - log1p(exp(-|x|))
        const float logsig = fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
        a[k] = expf(logsig * inv_tau);
      }
    }
    float* dst = out + (size_t)(t0 + tt) * channels + c;
    if constexpr (CH == 4) *reinterpret_cast<float4*>(dst) = make_float4(a[0], a[1], a[2], a[3]);
    else *dst = a[0];
  }
}

__device__ __forceinline__ void copy16(void* smem, const void* gmem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem) : "memory");
}
__device__ __forceinline__ void copy4(void* smem, const void* gmem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(s), "l"(gmem) : "memory");
}
__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copies_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// One block per (request, head, COLS value channels), KS * COLS threads.  KS (four or eight) lanes share a
// column of S (value channel j): lane part p keeps the key channels i with (i / 4) % KS == p, DK / KS of them
// (DK: the key size rounded up to 16, 32, 64, 128 or 256), and the sum over i of a token's S^T q meets
// by two or three shuffles.  Every warp reads the same staged q, k, a of CHUNK tokens, STAGES stages deep: while
// the block walks one chunk, the next three are on their way (a chunk's copies take longer than its
// arithmetic).  A token costs a block 3 DK / 4 shared-memory reads of 16 bytes a warp, which is what bounds
// a block of many warps; hence few columns a block, and more blocks.
// Lanes that share a column: four, or eight at key sizes from 64 on (a lane's share of the column, and with it the
// chain of additions a token, stays at most 32 long, and a block has several warps to hide the chain's waits behind).
__host__ __device__ constexpr int lanes_a_column(int dk) { return dk >= 64 ? 8 : 4; }
// Value channels a block: 32, or 16 where a step's blocks then still fit the GPU once (one prompt alone): the walk is a
// chain of dependent steps, and half the warps on twice the SMs walk it faster.
constexpr int COLS_WIDE = 32, COLS_NARROW = 16;
constexpr int STAGES = 4;

// MODE says what ``decay`` holds: DECAY_ROWS a row [heads * dim] per token (one number a key channel), DECAY_HEAD one
// constant per head (``heads`` numbers; a retention), DECAY_TOKEN one number per (token, head) for all of the head's
// key channels (a selective state space).  ``qk_heads``: q and k have that many heads (a divisor of ``heads``), head h
// reading q/k head h / (heads / qk_heads); the rows are [ q (qk_heads D) | k (qk_heads D) | v (heads V) | ... ].
// DECAY_BONUS: rows like DECAY_ROWS, and ``bonus`` [heads * dim] weighs the current token's k v^T in its own output.
// k stands ``k_offset`` numbers behind q, v ``v_offset``.
constexpr int DECAY_ROWS = 0, DECAY_HEAD = 1, DECAY_TOKEN = 2, DECAY_BONUS = 3;
template <int DK, bool VEC, int MODE, int COLS>
__global__ void __launch_bounds__(lanes_a_column(DK) * COLS)
gla_scan_kernel(const float* __restrict__ proj, int proj_stride, const float* __restrict__ decay,
                const int* __restrict__ req_indptr, const int* __restrict__ slots, float* __restrict__ state,
                float* __restrict__ out, int heads, int qk_heads, int dim, int vdim, int max_slots, float qscale,
                const float* __restrict__ bonus, long long k_offset, long long v_offset) {
  tl::pdl_launch_dependents();
  tl::pdl_wait();
  constexpr bool FIXED = MODE == DECAY_HEAD || MODE == DECAY_TOKEN;  // no decay row is staged
  constexpr int KS = lanes_a_column(DK);
  constexpr int PER = DK / KS;
  // a staged token: q, k, (a: only where the decay is a row a token), v, the token's decay number.  Without the a
  // row a stage holds twice as many tokens of the larger key sizes, and the walk meets half as many barriers.
  constexpr int VOFF = (FIXED ? 2 : 3) * DK;
  constexpr int CHUNK = FIXED ? (DK <= 128 ? 8 : 4) : (DK <= 64 ? 8 : (DK <= 128 ? 4 : 2));
  constexpr int row = VOFF + COLS + 4;
  __shared__ __align__(16) float stage[STAGES * CHUNK * row];  // [STAGES][CHUNK]
  constexpr int NT = KS * COLS;
  const int req = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int col0 = blockIdx.z * COLS;  // this block's value channels: col0 .. col0 + COLS
  const int cols_here = vdim - col0 < COLS ? vdim - col0 : COLS;
  const int part = tid % KS, col = col0 + tid / KS;
  const bool on = col < vdim;
  const int hv = heads * vdim;
  const int hq = h / (heads / qk_heads);  // the q/k head this head reads
  const int first = req_indptr[req], last = req_indptr[req + 1];
  const int slot = slots[req];
  const bool live = TL_DEBUG_OK(slot >= -1 && slot < max_slots, TL_DEBUG_SLOT, slot) && slot >= 0;
  if (!live) {  // a padding lane of a captured step: no state is touched
    if (part == 0 && on)
      for (int t = first; t < last; ++t) out[(size_t)t * hv + h * vdim + col] = 0.f;
    return;
  }
  // entries past dim (and past vdim) stay zero in both stages
  for (int e = tid; e < STAGES * CHUNK * row; e += NT) stage[e] = 0.f;
  __syncthreads();
  // which pieces of a chunk this thread copies: the same of every chunk, so the addresses are worked out once
  constexpr int PIECES = (CHUNK * ((FIXED ? 2 : 3) * DK / 4 + COLS / 4 + 1) + NT - 1) / NT;
  const float* piece_src[PIECES];
  int piece_to[PIECES], piece_token[PIECES];  // where in a stage; the token of the chunk (CHUNK: none)
  bool piece_decay[PIECES];
  if (VEC) {
    const int qd = dim >> 2, qv = cols_here >> 2, per_token = (FIXED ? 2 : 3) * qd + qv + (MODE == DECAY_TOKEN ? 1 : 0);
#pragma unroll
    for (int n = 0; n < PIECES; ++n) {
      const int e = tid + n * NT, tt = e / per_token, rest = e - tt * per_token;
      const int t = first + tt;
      piece_token[n] = tt < CHUNK ? tt : CHUNK;
      piece_decay[n] = false;
      if (rest < 2 * qd) {
        const int what = rest / qd, q4 = rest - what * qd;
        piece_src[n] = proj + (size_t)t * proj_stride + what * k_offset + hq * dim + 4 * q4;
        piece_to[n] = tt * row + what * DK + 4 * q4;
      } else if (!FIXED && rest < 3 * qd) {
        const int q4 = rest - 2 * qd;
        piece_src[n] = decay + (size_t)t * heads * dim + h * dim + 4 * q4;
        piece_to[n] = tt * row + 2 * DK + 4 * q4;
        piece_decay[n] = true;
      } else if (MODE == DECAY_TOKEN && rest == per_token - 1) {
        piece_src[n] = decay + (size_t)t * heads + h;
        piece_to[n] = tt * row + VOFF + COLS;
        piece_decay[n] = true;
      } else {
        const int q4 = rest - (FIXED ? 2 : 3) * qd;
        piece_src[n] = proj + (size_t)t * proj_stride + v_offset + h * vdim + col0 + 4 * q4;
        piece_to[n] = tt * row + VOFF + 4 * q4;
      }
    }
  }
  const size_t proj_step = (size_t)CHUNK * proj_stride, decay_step = (size_t)CHUNK * heads * (MODE == DECAY_TOKEN ? 1 : dim);
  auto fetch = [&](int base, int buf) {
    const int count = last - base < CHUNK ? last - base : CHUNK;
    float* dst = stage + (size_t)buf * CHUNK * row;
    if (VEC) {
#pragma unroll
      for (int n = 0; n < PIECES; ++n) {
        if (piece_token[n] < count) {
          if (MODE == DECAY_TOKEN && piece_decay[n]) copy4(dst + piece_to[n], piece_src[n]);
          else copy16(dst + piece_to[n], piece_src[n]);
        }
        piece_src[n] += (!FIXED || MODE == DECAY_TOKEN) && piece_decay[n] ? decay_step : proj_step;
      }
    } else {
      const int per_token = (FIXED ? 2 : 3) * dim + cols_here + (MODE == DECAY_TOKEN ? 1 : 0);
      for (int e = tid; e < count * per_token; e += NT) {
        const int tt = e / per_token, rest = e - tt * per_token;
        const int t = base + tt;
        const float* src;
        float* to;
        if (rest < 2 * dim) {
          const int what = rest / dim, i = rest - what * dim;
          src = proj + (size_t)t * proj_stride + what * k_offset + hq * dim + i;
          to = dst + tt * row + what * DK + i;
        } else if (!FIXED && rest < 3 * dim) {
          const int i = rest - 2 * dim;
          src = decay + (size_t)t * heads * dim + h * dim + i;
          to = dst + tt * row + 2 * DK + i;
        } else if (MODE == DECAY_TOKEN && rest == per_token - 1) {
          src = decay + (size_t)t * heads + h;
          to = dst + tt * row + VOFF + COLS;
        } else {
          const int i = rest - (FIXED ? 2 : 3) * dim;
          src = proj + (size_t)t * proj_stride + v_offset + h * vdim + col0 + i;
          to = dst + tt * row + VOFF + i;
        }
        copy4(to, src);
      }
    }
    copies_commit();
  };
  for (int s = 0; s < STAGES - 1; ++s) {  // always STAGES - 1 groups in flight (some of them empty)
    if (first + s * CHUNK < last) fetch(first + s * CHUNK, s);
    else copies_commit();
  }

  // this lane's key channels: i = 4 (n / 4 * KS + part) + n % 4
  float* mine = state + ((size_t)slot * heads + h) * dim * vdim;
  float S[PER];
#pragma unroll
  for (int n = 0; n < PER; ++n) {
    const int i = 4 * ((n >> 2) * KS + part) + (n & 3);
    S[n] = (on && i < dim) ? mine[(size_t)i * vdim + col] : 0.f;
  }

  float U[MODE == DECAY_BONUS ? PER : 1];  // the bonus of the same key channels
  if (MODE == DECAY_BONUS) {
#pragma unroll
    for (int n = 0; n < PER; ++n) {
      const int i = 4 * ((n >> 2) * KS + part) + (n & 3);
      U[n] = i < dim ? bonus[(size_t)h * dim + i] : 0.f;
    }
  }

  const float head_decay = MODE == DECAY_HEAD ? decay[h] : 0.f;
  int buf = 0;
  for (int base = first; base < last; base += CHUNK, buf = (buf + 1) % STAGES) {
    const int count = last - base < CHUNK ? last - base : CHUNK;
    // the stage that the chunk before this one used is free (the barrier at the end of its walk)
    if (base + (STAGES - 1) * CHUNK < last) fetch(base + (STAGES - 1) * CHUNK, (buf + STAGES - 1) % STAGES);
    else copies_commit();
    copies_wait<STAGES - 1>();  // all but the newest STAGES - 1 groups: this chunk has landed
    __syncthreads();
    const float* chunk = stage + (size_t)buf * CHUNK * row;
    auto walk = [&](int tt) {
      const float* tok = chunk + tt * row;
      const float4* q4 = reinterpret_cast<const float4*>(tok);
      const float4* k4 = reinterpret_cast<const float4*>(tok + DK);
      const float4* a4 = reinterpret_cast<const float4*>(tok + 2 * DK);
      const float v = tok[VOFF + (on ? col - col0 : 0)];
      const float fixed = MODE == DECAY_TOKEN ? tok[VOFF + COLS] : head_decay;
      float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
      for (int n = 0; n < PER / 4; ++n) {
        const float4 a = FIXED ? make_float4(fixed, fixed, fixed, fixed) : a4[n * KS + part];
        const float4 k = k4[n * KS + part], q = q4[n * KS + part];
        if constexpr (MODE == DECAY_BONUS) {  // the output reads the state before the token joins it
          const float kx = k.x * v, ky = k.y * v, kz = k.z * v, kw = k.w * v;
          o0 = fmaf(q.x, fmaf(U[4 * n], kx, S[4 * n]), o0);
          o1 = fmaf(q.y, fmaf(U[4 * n + 1], ky, S[4 * n + 1]), o1);
          o2 = fmaf(q.z, fmaf(U[4 * n + 2], kz, S[4 * n + 2]), o2);
          o3 = fmaf(q.w, fmaf(U[4 * n + 3], kw, S[4 * n + 3]), o3);
          S[4 * n] = fmaf(a.x, S[4 * n], kx);
          S[4 * n + 1] = fmaf(a.y, S[4 * n + 1], ky);
          S[4 * n + 2] = fmaf(a.z, S[4 * n + 2], kz);
          S[4 * n + 3] = fmaf(a.w, S[4 * n + 3], kw);
          continue;
        }
        S[4 * n] = fmaf(k.x, v, a.x * S[4 * n]);
        S[4 * n + 1] = fmaf(k.y, v, a.y * S[4 * n + 1]);
        S[4 * n + 2] = fmaf(k.z, v, a.z * S[4 * n + 2]);
        S[4 * n + 3] = fmaf(k.w, v, a.w * S[4 * n + 3]);
        o0 = fmaf(q.x, S[4 * n], o0);
        o1 = fmaf(q.y, S[4 * n + 1], o1);
        o2 = fmaf(q.z, S[4 * n + 2], o2);
        o3 = fmaf(q.w, S[4 * n + 3], o3);
      }
      float o = (o0 + o1) + (o2 + o3);
      o += __shfl_xor_sync(0xffffffffu, o, 1);
      o += __shfl_xor_sync(0xffffffffu, o, 2);
      if (KS == 8) o += __shfl_xor_sync(0xffffffffu, o, 4);
      if (on && part == 0) out[(size_t)(base + tt) * hv + h * vdim + col] = o * qscale;
    };
    // A whole chunk: the next token's shared-memory reads are under way while this one's arithmetic runs, and the lanes'
    // shares of all the chunk's outputs meet together, in CHUNK independent shuffles a round.  (Key sizes whose share of a
    // token would not fit the registers twice walk token by token.)
    if (PER <= 16 && count == CHUNK) {
      constexpr int QD = PER <= 16 ? PER / 4 : 1;
      float4 Q[2][QD], K[2][QD], A[2][QD];
      float V[2], F[2];
      auto load = [&](int tt, int w) {
        const float* tok = chunk + tt * row;
        const float4* q4 = reinterpret_cast<const float4*>(tok);
        const float4* k4 = reinterpret_cast<const float4*>(tok + DK);
        const float4* a4 = reinterpret_cast<const float4*>(tok + 2 * DK);
        V[w] = tok[VOFF + (on ? col - col0 : 0)];
        F[w] = MODE == DECAY_TOKEN ? tok[VOFF + COLS] : head_decay;
#pragma unroll
        for (int n = 0; n < QD; ++n) {
          Q[w][n] = q4[n * KS + part];
          K[w][n] = k4[n * KS + part];
          if (!FIXED) A[w][n] = a4[n * KS + part];
        }
      };
      float O[CHUNK];
      load(0, 0);
#pragma unroll
      for (int tt = 0; tt < CHUNK; ++tt) {
        const int w = tt & 1;
        if (tt + 1 < CHUNK) load(tt + 1, w ^ 1);
        const float v = V[w];
        float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
        for (int n = 0; n < QD; ++n) {
          const float4 k = K[w][n], q = Q[w][n];
          const float4 a = FIXED ? make_float4(F[w], F[w], F[w], F[w]) : A[w][n];
          if constexpr (MODE == DECAY_BONUS) {
            const float kx = k.x * v, ky = k.y * v, kz = k.z * v, kw = k.w * v;
            o0 = fmaf(q.x, fmaf(U[4 * n], kx, S[4 * n]), o0);
            o1 = fmaf(q.y, fmaf(U[4 * n + 1], ky, S[4 * n + 1]), o1);
            o2 = fmaf(q.z, fmaf(U[4 * n + 2], kz, S[4 * n + 2]), o2);
            o3 = fmaf(q.w, fmaf(U[4 * n + 3], kw, S[4 * n + 3]), o3);
            S[4 * n] = fmaf(a.x, S[4 * n], kx);
            S[4 * n + 1] = fmaf(a.y, S[4 * n + 1], ky);
            S[4 * n + 2] = fmaf(a.z, S[4 * n + 2], kz);
            S[4 * n + 3] = fmaf(a.w, S[4 * n + 3], kw);
          } else {
            S[4 * n] = fmaf(k.x, v, a.x * S[4 * n]);
            S[4 * n + 1] = fmaf(k.y, v, a.y * S[4 * n + 1]);
            S[4 * n + 2] = fmaf(k.z, v, a.z * S[4 * n + 2]);
            S[4 * n + 3] = fmaf(k.w, v, a.w * S[4 * n + 3]);
            o0 = fmaf(q.x, S[4 * n], o0);
            o1 = fmaf(q.y, S[4 * n + 1], o1);
            o2 = fmaf(q.z, S[4 * n + 2], o2);
            o3 = fmaf(q.w, S[4 * n + 3], o3);
          }
        }
        O[tt] = (o0 + o1) + (o2 + o3);
      }
#pragma unroll
      for (int m = 1; m < KS; m <<= 1)
#pragma unroll
        for (int tt = 0; tt < CHUNK; ++tt) O[tt] += __shfl_xor_sync(0xffffffffu, O[tt], m);
#pragma unroll
      for (int tt = 0; tt < CHUNK; ++tt)
        if (on && part == tt % KS) out[(size_t)(base + tt) * hv + h * vdim + col] = O[tt] * qscale;
    } else {
      for (int tt = 0; tt < count; ++tt) walk(tt);
    }
    __syncthreads();  // the stage is free for the chunk after the next
  }
  if (on) {
#pragma unroll
    for (int n = 0; n < PER; ++n) {
      const int i = 4 * ((n >> 2) * KS + part) + (n & 3);
      if (i < dim) mine[(size_t)i * vdim + col] = S[n];
    }
  }
}

constexpr int FINISH_WARPS = 4;

template <typename T>
__global__ void __launch_bounds__(FINISH_WARPS * 32)
gla_finish_kernel(const float* __restrict__ o, const float* __restrict__ proj, int proj_stride, int gate_offset,
                  const float* __restrict__ weight, int weight_stride, T* __restrict__ out, long long items, int heads, int vdim,
                  float eps) {
  tl::pdl_launch_dependents();
  tl::pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * FINISH_WARPS + warp;
  if (item >= items) return;
  const long long t = item / heads;
  const int h = (int)(item % heads);
  const int hv = heads * vdim;
  const float* row = o + (size_t)t * hv + h * vdim;
  float ss = 0.f;
  for (int i = lane; i < vdim; i += 32) ss = fmaf(row[i], row[i], ss);
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / (float)vdim + eps);
  const float* gate = proj + (size_t)t * proj_stride + gate_offset + h * vdim;
  for (int i = lane; i < vdim; i += 32) {
    const float g = gate[i];
    out[(size_t)t * hv + h * vdim + i] = from_float<T>(row[i] * inv * (weight ? weight[h * weight_stride + i] : 1.f) * (g / (1.f + expf(-g))));
  }
}

// The same with LANES lanes an item, four neighbouring entries a lane at a time (vdim a multiple of 4, everything 16-byte
// aligned): a warp takes 32 / LANES heads at once.
template <typename T, int LANES>
__global__ void __launch_bounds__(FINISH_WARPS * 32)
gla_finish_wide_kernel(const float* __restrict__ o, const float* __restrict__ proj, int proj_stride, int gate_offset,
                       const float* __restrict__ weight, int weight_stride, T* __restrict__ out, long long items, int heads,
                       int vdim, float eps) {
  tl::pdl_launch_dependents();
  tl::pdl_wait();
  constexpr int KEEP = LANES == 32 ? 2 : 1;  // quads of a lane: vdim up to 4 LANES KEEP
  const int sub = threadIdx.x % LANES;
  const long long item = ((long long)blockIdx.x * FINISH_WARPS * 32 + threadIdx.x) / LANES;
  const bool live = item < items;
  const long long t = live ? item / heads : 0;
  const int h = live ? (int)(item % heads) : 0;
  const int hv = heads * vdim;
  const float* row = o + (size_t)t * hv + h * vdim;
  const float* gate = proj + (size_t)t * proj_stride + gate_offset + h * vdim;
  float4 v[KEEP], g[KEEP];
  float ss = 0.f;
#pragma unroll
  for (int n = 0; n < KEEP; ++n) {
    const int i = (sub + n * LANES) * 4;
    v[n] = g[n] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live && i < vdim) {
      v[n] = *reinterpret_cast<const float4*>(row + i);
      g[n] = *reinterpret_cast<const float4*>(gate + i);
    }
    ss = fmaf(v[n].x, v[n].x, ss);
    ss = fmaf(v[n].y, v[n].y, ss);
    ss = fmaf(v[n].z, v[n].z, ss);
    ss = fmaf(v[n].w, v[n].w, ss);
  }
#pragma unroll
  for (int m = LANES / 2; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  const float inv = 1.f / sqrtf(ss / (float)vdim + eps);
#pragma unroll
  for (int n = 0; n < KEEP; ++n) {
    const int i = (sub + n * LANES) * 4;
    if (!live || i >= vdim) continue;
    float4 w = make_float4(1.f, 1.f, 1.f, 1.f);
    if (weight) w = *reinterpret_cast<const float4*>(weight + h * weight_stride + i);
    const float r[4] = {v[n].x * inv * w.x * (g[n].x / (1.f + expf(-g[n].x))), v[n].y * inv * w.y * (g[n].y / (1.f + expf(-g[n].y))),
                        v[n].z * inv * w.z * (g[n].z / (1.f + expf(-g[n].z))), v[n].w * inv * w.w * (g[n].w / (1.f + expf(-g[n].w)))};
    T* dst = out + (size_t)t * hv + h * vdim + i;
    if constexpr (sizeof(T) == 4) {
      *reinterpret_cast<float4*>(dst) = make_float4(r[0], r[1], r[2], r[3]);
    } else {
      const __nv_bfloat162 lo = __floats2bfloat162_rn(r[0], r[1]), hi = __floats2bfloat162_rn(r[2], r[3]);
      *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
    }
  }
}

// Split-half rotation of the first ``dims`` entries of ``heads`` consecutive heads of ``dim`` entries in float32
// rows, in place: entry i (< dims / 2) pairs with i + dims / 2, angle = float(position) * inv_freq[i].
__global__ void rotate_heads_kernel(float* __restrict__ rows, int stride, const int* __restrict__ positions,
                                    const float* __restrict__ inv_freq, int heads, int dim, int half, size_t total) {
  tl::pdl_launch_dependents();
  tl::pdl_wait();
  const size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= total) return;
  const int i = (int)(e % half);
  const int h = (int)((e / half) % heads);
  const size_t t = e / ((size_t)half * heads);
  float s, c;
  sincosf((float)positions[t] * inv_freq[i], &s, &c);
  float* head = rows + t * stride + (size_t)h * dim;
  const float u = head[i], v = head[i + half];
  head[i] = u * c - v * s;
  head[i + half] = v * c + u * s;
}

}  // namespace

TL_DEBUG_READER(tl_gla_debug_error)

extern "C" {

// decay: float32 [tokens, channels] scratch; w2t: [rank, channels]; the low-rank input is
// proj[t, low_offset : low_offset + rank].  tau > 0: sigmoid(W2 l + bias)^(1 / tau); 0: exp(-exp(W2 tanh(l) + bias)).
int tl_gla_decay(const float* proj, int proj_stride, int low_offset, const float* w2t, const float* bias, float* decay,
                 int tokens, int channels, int rank, float tau, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (channels <= 0 || rank <= 0 || rank > 1024 || !(tau >= 0.f)) return TL_ERR_UNSUPPORTED;
  const int chunks = (tokens + DECAY_TOKENS - 1) / DECAY_TOKENS;
  const bool four = chunks >= 64 && channels % 4 == 0 && (((uintptr_t)w2t | (uintptr_t)decay) & 15) == 0;
  const int per_block = DECAY_NT * (four ? 4 : 1);
  const dim3 grid(chunks, (channels + per_block - 1) / per_block);
  if (grid.y > 65535) return TL_ERR_UNSUPPORTED;
  const size_t smem = (size_t)DECAY_TOKENS * ((rank + 3) & ~3) * sizeof(float);
#define TL_DECAY(TANH, CH)                                                                                             \
  tl::launch_kernel(gla_decay_kernel<TANH, CH>, grid, DECAY_NT, smem, stream, proj, proj_stride, low_offset, w2t, bias, decay, \
                    tokens, channels, rank, tau > 0.f ? 1.f / tau : 0.f)
  if (tau > 0.f && four) TL_DECAY(false, 4);
  else if (tau > 0.f) TL_DECAY(false, 1);
  else if (four) TL_DECAY(true, 4);
  else TL_DECAY(true, 1);
#undef TL_DECAY
  return TL_LAUNCH_CHECK();
}

// state: float32 [max_slots, heads, dim, vdim]; out: float32 [tokens, heads * vdim].
// decay_mode: 0 ``decay`` holds [tokens, heads * dim] rows, 1 one constant per head, 2 [tokens, heads] (one number per
// token and head), 3 rows and ``bonus`` [heads * dim].  k_offset, v_offset: how far k and v stand behind q.  qk_heads: how many heads q and k have (divides heads).
int tl_gla_scan(const float* proj, int proj_stride, const float* decay, const int* req_indptr, const int* slots,
                float* state, float* out, int requests, int heads, int qk_heads, int dim, int vdim, int max_slots,
                float qscale, int decay_mode, const float* bonus, long long k_offset, long long v_offset,
                cudaStream_t stream) {
  if (requests <= 0) return 0;
  if (dim <= 0 || dim > 256 || vdim <= 0 || vdim > 256 || heads > 65535) return TL_ERR_UNSUPPORTED;
  if (qk_heads <= 0 || heads % qk_heads || decay_mode < 0 || decay_mode > 3) return TL_ERR_UNSUPPORTED;
  if ((decay_mode == DECAY_BONUS) != (bonus != nullptr)) return TL_ERR_UNSUPPORTED;
  const bool fixed_decay = decay_mode == DECAY_HEAD || decay_mode == DECAY_TOKEN;
  const bool vec = dim % 4 == 0 && vdim % 4 == 0 && proj_stride % 4 == 0 && k_offset % 4 == 0 && v_offset % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(proj) & 15) == 0 &&
                   (fixed_decay || (reinterpret_cast<uintptr_t>(decay) & 15) == 0);
  static int sms = 0;
  if (!sms) {
    int device = 0;
    cudaGetDevice(&device);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device);
  }
  const bool narrow = vec && (long long)requests * heads * ((vdim + COLS_NARROW - 1) / COLS_NARROW) <= sms;
#define TL_SCAN_ONE(DK, VEC, MODE, COLS)                                                                                   \
  tl::launch_kernel(gla_scan_kernel<DK, VEC, MODE, COLS>, dim3(requests, heads, (vdim + COLS - 1) / COLS),                 \
                    lanes_a_column(DK) * COLS, 0, stream, proj, proj_stride, decay, req_indptr, slots, state, out, heads,  \
                    qk_heads, dim, vdim, max_slots, qscale, bonus, k_offset, v_offset)
#define TL_SCAN_MODE(DK, MODE)                                    \
  {                                                               \
    if (narrow) TL_SCAN_ONE(DK, true, MODE, COLS_NARROW);         \
    else if (vec) TL_SCAN_ONE(DK, true, MODE, COLS_WIDE);         \
    else TL_SCAN_ONE(DK, false, MODE, COLS_WIDE);                 \
  }
#define TL_SCAN(DK)                                                    \
  {                                                                    \
    if (decay_mode == DECAY_HEAD) TL_SCAN_MODE(DK, DECAY_HEAD)         \
    else if (decay_mode == DECAY_TOKEN) TL_SCAN_MODE(DK, DECAY_TOKEN)  \
    else if (decay_mode == DECAY_BONUS) TL_SCAN_MODE(DK, DECAY_BONUS)  \
    else TL_SCAN_MODE(DK, DECAY_ROWS)                                  \
  }
  if (dim <= 16) TL_SCAN(16)
  else if (dim <= 32) TL_SCAN(32)
  else if (dim <= 64) TL_SCAN(64)
  else if (dim <= 128) TL_SCAN(128)
  else TL_SCAN(256)
#undef TL_SCAN
#undef TL_SCAN_MODE
#undef TL_SCAN_ONE
  return TL_LAUNCH_CHECK();
}

int tl_rotate_heads_f32(float* rows, int stride, const int* positions, const float* inv_freq, int tokens, int heads,
                        int dim, int dims, cudaStream_t stream) {
  if (tokens <= 0 || dims <= 0) return 0;
  if (dims % 2 || dims > dim || heads <= 0) return TL_ERR_UNSUPPORTED;
  const size_t total = (size_t)tokens * heads * (dims / 2);
  tl::launch_kernel(rotate_heads_kernel, (unsigned)((total + 255) / 256), 256, 0, stream, rows, stride, positions,
                    inv_freq, heads, dim, dims / 2, total);
  return TL_LAUNCH_CHECK();
}

int tl_gla_finish(const float* o, const float* proj, int proj_stride, int gate_offset, const float* weight, int weight_stride, void* out,
                  int out_dtype, int tokens, int heads, int vdim, float eps, cudaStream_t stream) {
  const long long items = (long long)tokens * heads;
  if (items <= 0) return 0;
  const uintptr_t all = (uintptr_t)o | (uintptr_t)(proj + gate_offset) | (uintptr_t)weight | (uintptr_t)out;
  if (vdim % 4 == 0 && vdim <= 256 && proj_stride % 4 == 0 && (all & 15) == 0) {
#define TL_FINISH_WIDE(T, LANES)                                                                                        \
  tl::launch_kernel(gla_finish_wide_kernel<T, LANES>, (unsigned)((items * LANES + FINISH_WARPS * 32 - 1) / (FINISH_WARPS * 32)), \
                    FINISH_WARPS * 32, 0, stream, o, proj, proj_stride, gate_offset, weight, weight_stride, (T*)out, items, heads, \
                    vdim, eps)
    if (out_dtype == TL_DTYPE_F32) {
      if (vdim <= 32) TL_FINISH_WIDE(float, 8);
      else if (vdim <= 64) TL_FINISH_WIDE(float, 16);
      else TL_FINISH_WIDE(float, 32);
    } else {
      if (vdim <= 32) TL_FINISH_WIDE(__nv_bfloat16, 8);
      else if (vdim <= 64) TL_FINISH_WIDE(__nv_bfloat16, 16);
      else TL_FINISH_WIDE(__nv_bfloat16, 32);
    }
#undef TL_FINISH_WIDE
    return TL_LAUNCH_CHECK();
  }
  const unsigned blocks = (unsigned)((items + FINISH_WARPS - 1) / FINISH_WARPS);
  if (out_dtype == TL_DTYPE_F32)
    tl::launch_kernel(gla_finish_kernel<float>, blocks, FINISH_WARPS * 32, 0, stream, o, proj, proj_stride,
                      gate_offset, weight, weight_stride, (float*)out, items, heads, vdim, eps);
  else
    tl::launch_kernel(gla_finish_kernel<__nv_bfloat16>, blocks, FINISH_WARPS * 32, 0, stream, o, proj, proj_stride,
                      gate_offset, weight, weight_stride, (__nv_bfloat16*)out, items, heads, vdim, eps);
  return TL_LAUNCH_CHECK();
}

}  // extern "C"
