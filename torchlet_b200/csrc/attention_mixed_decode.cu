// Paged attention of SINGLE TOKENS, bfloat16 on the tensor cores, for scores that are mixed across the heads before the
// softmax (s_h <- sum_g T[h, g] s_g) and a sliding window that may keep the sequence's first tokens.  Head rows of P = 64 or
// 128 entries, up to 16 query heads a KV head.
//
// Mixing needs the scores of ALL heads with a key at once, so one CTA takes all heads of a request over a share of its key
// tiles (blockIdx.y; the last CTA of a request to finish merges the shares), and every key and value row is read once:
//
//   keys and values  tiles of BN = 16, 32 or 64 absolute positions (as many as keep a tile at 64 KB or less), K and V of all
//                    KV heads, by TMA: 3-D boxes of 64 entries x positions of a page x KV heads (128-byte swizzle), into a
//                    ring for K and one for V, filled by a loader warp each; first the tiles of kept positions that lie
//                    wholly before the window, then the window's
//   scores           S^T [keys x heads of a group] = K Q^T a KV head, mma.sync m16n8k16 with the keys as rows: a group of up
//                    to eight heads fills one column tile; the float32 scores go to shared memory
//   softmax          a warp takes two heads at a time: the mixed score of a key a lane, float32, running max and sum
//   values           O^T [entries x heads of a group] += V^T P^T, 16 entries of one KV head a warp and unit, accumulators in
//                    registers for the whole walk
//
// A tile's three phases are chains of short dependent steps, so they run on three groups of eight warps as a pipeline: while
// one group multiplies the scores of tile t, the next is in the softmax of tile t - 1 and the third adds the values of tile
// t - 2, with one barrier a step (one group that did all three in turn took 2.4 us a tile).
//
// (Spreading the mixed queries over all KV heads, as the prompt kernel does, would multiply every head with every KV head's
// keys; here each head is multiplied with its own, and the mixing is H x H multiplications a key.)
// Waits are bounded (tcgen05.cuh); one that gives up leaves a code that tl_attention_mixed_decode_error() returns.
#include <math.h>
#include <string.h>

#include <mutex>
#include <unordered_map>

#include "common.cuh"
#include "tcgen05.cuh"

namespace {

using namespace tl;

constexpr int GROUP = 8;               // warps of each of the three compute groups
constexpr int COMPUTE = 3 * GROUP * 32;
constexpr int THREADS = COMPUTE + 64;  // two more warps load
constexpr int MAX_SLOTS = 4;           // tiles a ring holds
constexpr int MAX_HEADS = 64;
constexpr int TILE_LIMIT = 64 * 1024;  // bytes of a tile, K and V
constexpr int SMEM_LIMIT = 232448;

__device__ int g_error_word = 0;

struct Params {
  const __nv_bfloat16* q;  // [tokens][q_stride]: head h at h * P
  long long q_stride;
  const int* block_table;
  int table_width;
  const int *req_indptr, *kv_before, *tile_req;  // tile_req null: tile i is request i
  __nv_bfloat16* out;                            // [tokens][out_stride]: head h at h * v_cols
  long long out_stride;
  float *part_acc, *part_ml;  // [tiles][splits][H][P], [tiles][splits][H][2]
  int* arrivals;              // [tiles], zero between launches
  int H, G, page_shift, window, keep, v_cols, splits;
  int slots;          // tiles a ring holds: as many as fit, 2 to 4
  int bn, box_shift;  // keys a tile; log2 of the positions a box holds
  const float* talk;  // [H][H] or null: no mixing
  float scale_log2;
  int num_pages;
};

__device__ __forceinline__ void ldmatrix_x4(unsigned (&r)[4], const void* smem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(s));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned (&r)[4], const void* smem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(s));
}
__device__ __forceinline__ void mma_16816(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// 2^x by the special-function unit (ex2.approx: 2 ulp; the weights are rounded to bfloat16 anyway).
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Barrier of the compute warps alone.
__device__ __forceinline__ void compute_sync() { asm volatile("bar.sync 1, %0;" ::"n"(COMPUTE) : "memory"); }

// The key tiles of a request: ``kept`` tiles from position 0 on, then the tiles from ``first`` on.
struct Walk {
  int kept, first, count, lo, hi, keep, bn;
  __device__ __forceinline__ Walk(const Params& p, int pos) {
    bn = p.bn;
    keep = p.keep;
    hi = pos;
    lo = first_key(pos, p.window);
    first = lo / bn;
    kept = min((keep + bn - 1) / bn, first);
    count = kept + hi / bn + 1 - first;
  }
  __device__ __forceinline__ int tile(int i) const { return i < kept ? i : first + (i - kept); }
  __device__ __forceinline__ bool dead(int key) const { return key > hi || (key < lo && key >= keep); }
  __device__ __forceinline__ bool edge(int i) const {
    const int k0 = tile(i) * bn, k1 = k0 + bn - 1;
    return k1 > hi || max(k0, keep) <= min(k1, lo - 1);
  }
  // tiles a CTA takes, with ``splits`` CTAs in the grid: no share below 96 keys (three tiles of 32: at batch 8 and 17 shares
  // of two tiles 12.5 us, with 12 of three 11.5 us)
  __device__ __forceinline__ int share(int splits) const { return max((96 + bn - 1) / bn, (count + splits - 1) / splits); }
};

// NT: column tiles of eight heads a group; MAXU: units of 16 value entries a value warp accumulates; WIDE: tiles of 64 keys
// (else 16 or 32).  The loops are bound by the instructions they issue, so what does not change from tile to tile (a lane's
// offsets in a tile) is worked out once, and the rows of scores and weights have compile-time strides.
template <int P, int NT, int MAXU, bool WIDE>
__global__ void __launch_bounds__(THREADS, 1)
attention_mixed_decode_kernel(const __grid_constant__ CUtensorMap map_kv, const Params p) {
  constexpr int SLABS = P / 64;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int bn = p.bn, H = p.H, G = p.G, gs = H / G;
  const int slab_elems = G * bn * 64, slot_elems = SLABS * slab_elems;  // a tile's keys, or its values
  __nv_bfloat16* k_ring = reinterpret_cast<__nv_bfloat16*>(base);
  __nv_bfloat16* v_ring = k_ring + p.slots * slot_elems;
  constexpr int ps_stride = WIDE ? 72 : 40, ss_stride = WIDE ? 68 : 36;
  const int ps_elems = (H + 16) * ps_stride, ss_elems = H * ss_stride;
  __nv_bfloat16* ps = v_ring + p.slots * slot_elems;                    // two of [H + 16][ps_stride]
  float* ss = reinterpret_cast<float*>(ps + 2 * ps_elems);              // two of [H][ss_stride]
  float* talk = ss + 2 * ss_elems;                                      // [H][H]
  float* m_run = talk + (p.talk ? H * H : 0);                           // [H]
  float* l_run = m_run + H;                                             // [H]
  float* corr = l_run + H;                                              // two of [H + 16]
  uint64_t* k_full = reinterpret_cast<uint64_t*>((reinterpret_cast<uintptr_t>(corr + 2 * (H + 16)) + 7) & ~(uintptr_t)7);
  uint64_t* v_full = k_full + MAX_SLOTS;
  uint64_t* k_empty = v_full + MAX_SLOTS;  // (GROUP arrivals: one a warp of the group that reads it)
  uint64_t* v_empty = k_empty + MAX_SLOTS;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(v_empty + MAX_SLOTS);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tile_index = blockIdx.x, split = blockIdx.y;
  const int req = p.tile_req ? p.tile_req[tile_index] : tile_index;
  const int before = p.kv_before[req];
  const int token = p.req_indptr[req];
  const int* table = p.block_table + (size_t)req * p.table_width;
  const Walk walk(p, before);
  const int per = walk.share(p.splits), my_splits = (walk.count + per - 1) / per;
  if (split >= my_splits) {  // the request is too short to need this CTA
    pdl_wait();
    return;
  }
  const int begin = split * per, count = min(per, walk.count - begin);

  if (threadIdx.x == 0) {
    for (int i = 0; i < p.slots; ++i) {
      tc::mbar_init(&k_full[i], 1);
      tc::mbar_init(&v_full[i], 1);
      tc::mbar_init(&k_empty[i], GROUP);
      tc::mbar_init(&v_empty[i], GROUP);
    }
    *abort_flag = 0;
    tc::mbar_fence_init();
    tc::prefetch_tensormap(&map_kv);
  }
  __syncthreads();

  if (warp >= 3 * GROUP) {
    // ------------------------------------------------------------ loaders: one warp for K, one for V; one lane a box
    const int plane = warp - 3 * GROUP;
    __nv_bfloat16* ring = plane ? v_ring : k_ring;
    uint64_t *full = plane ? v_full : k_full, *empty = plane ? v_empty : k_empty;
    const int box = 1 << p.box_shift, boxes_per_tile = bn >> p.box_shift;
    bool waited = false;
    int slot = 0;
    uint32_t phase = 0;
    for (int index = 0; index < count; ++index) {
      const int key0 = walk.tile(begin + index) * bn;
      // tiles that earlier steps wrote may be requested before the wait on the preceding kernel
      if (!waited && (key0 + bn - 1 >= before || index == p.slots)) {
        pdl_wait();
        waited = true;
      }
      tc::mbar_wait(&empty[slot], phase ^ 1, abort_flag, &g_error_word, 2);
      if (lane == 0) tc::mbar_expect_tx(&full[slot], (uint32_t)slot_elems * 2);
      __syncwarp();
      for (int b = lane; b < SLABS * boxes_per_tile; b += 32) {
        const int part = b % boxes_per_tile, slab = b / boxes_per_tile;
        const int key = key0 + part * box, entry = key >> p.page_shift;
        int page = (entry < p.table_width && key <= walk.hi) ? table[entry] : 0;  // beyond the last key: page 0, always there
        if (!TL_DEBUG_OK(page >= 0 && page < p.num_pages, TL_DEBUG_PAGE, page)) page = 0;
        tc::tma_load_3d(ring + slot * slot_elems + slab * slab_elems + part * (G * box * 64), &map_kv, &full[slot], slab * 64,
                        key & ((1 << p.page_shift) - 1), (page * 2 + plane) * G);
      }
      if (++slot == p.slots) {
        slot = 0;
        phase ^= 1;
      }
    }
    if (!waited) pdl_wait();
    pdl_launch_dependents();
    return;
  }

  // What the step's kernels do not write does not have to wait for them.  The rows behind the last head fill a group's column
  // tile: their columns are computed and never used, but must not be read before they hold something.
  for (int i = threadIdx.x; i < 16 * ps_stride; i += COMPUTE)
    ps[H * ps_stride + i] = ps[ps_elems + H * ps_stride + i] = __float2bfloat16_rn(0.f);
  if (p.talk)
    for (int i = threadIdx.x; i < H * H; i += COMPUTE) talk[i] = p.talk[i];
  for (int i = threadIdx.x; i < 16; i += COMPUTE) corr[H + i] = corr[2 * H + 16 + i] = 0.f;
  for (int i = threadIdx.x; i < H; i += COMPUTE) {
    m_run[i] = -INFINITY;
    l_run[i] = 0.f;
  }
  const int blocks = (p.v_cols + 15) / 16;  // units of 16 value entries a KV head
  const int units = G * blocks;
  const int key_blocks = bn >> 4;
  const int group = warp / GROUP, member = warp - group * GROUP;
  // A slab's rows are [boxes][KV heads][8 or 16 positions]: where this lane's key of a 16-key block lies (ldmatrix takes keys
  // (lane & 7) + 8 upper, ``upper`` a bit of the lane), and how far the next 16-key block is.  All in elements.
  const int box = 1 << p.box_shift, block_step = G * 16 * 64;
  auto lane_row = [&](int upper) { return ((lane & 7) + (box == 16 ? upper * 8 : upper * G * 8)) * 64; };
  const __nv_bfloat16* q_row = p.q + (size_t)token * p.q_stride;
  int slot = 0;
  uint32_t phase = 0;
  pdl_wait();
  pdl_launch_dependents();

  // Step t: the first group computes the scores of tile t, the second the softmax of tile t - 1, the third adds the values of
  // tile t - 2; one barrier a step.
  if (group == 0) {
    // ---- scores: S^T of 16 keys x the heads of one KV head a unit.  Up to eight KV heads a warp keeps to one of them, whose
    // queries stay in its registers (the operand's columns beyond the group's heads are zero).
    const bool fixed = G <= GROUP;
    const int warps_a_head = fixed ? GROUP / G : 1;
    const int mine = member / warps_a_head;  // (fixed) the KV head; beyond the last: no work
    unsigned q_frag[P / 16][NT][2];
    auto load_queries = [&](int c) {
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int head = n * 8 + (lane >> 2);
        const __nv_bfloat16* at = q_row + (size_t)(c * gs + head) * P + (lane & 3) * 2;
#pragma unroll
        for (int k = 0; k < P / 16; ++k) {
          q_frag[k][n][0] = head < gs ? *reinterpret_cast<const unsigned*>(at + k * 16) : 0u;
          q_frag[k][n][1] = head < gs ? *reinterpret_cast<const unsigned*>(at + k * 16 + 8) : 0u;
        }
      }
    };
    if (fixed && mine < G) load_queries(mine);
    int key_chunk[4];  // the four 16-entry slices of a slab, as this lane reads them
#pragma unroll
    for (int k = 0; k < 4; ++k) key_chunk[k] = lane_row((lane >> 3) & 1) + (((2 * k + (lane >> 4)) ^ (lane & 7)) << 3);
    compute_sync();
    for (int index = 0; index < count; ++index) {
      float* s_out = ss + (index & 1) * ss_elems;
      const __nv_bfloat16* keys = k_ring + slot * slot_elems;
      tc::mbar_wait(&k_full[slot], phase, abort_flag, &g_error_word, 1);
      for (int c = fixed ? mine : member; c < G; c += GROUP) {
        if (!fixed) load_queries(c);
        for (int kb = fixed ? member - mine * warps_a_head : 0; kb < key_blocks; kb += warps_a_head) {
          float s[2][NT][4];
#pragma unroll
          for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[0][n][e] = s[1][n][e] = 0.f;
          const __nv_bfloat16* kblock = keys + kb * block_step + c * box * 64;
#pragma unroll
          for (int k = 0; k < P / 16; ++k) {
            unsigned a[4];
            ldmatrix_x4(a, kblock + (k >> 2) * slab_elems + key_chunk[k & 3]);
#pragma unroll
            for (int n = 0; n < NT; ++n) mma_16816(s[k & 1][n], a, q_frag[k][n][0], q_frag[k][n][1]);
          }
          float* at = s_out + (c * gs + (lane & 3) * 2) * ss_stride + kb * 16 + (lane >> 2);
#pragma unroll
          for (int n = 0; n < NT; ++n) {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              if (n * 8 + (lane & 3) * 2 + e < gs) {
                at[(n * 8 + e) * ss_stride] = s[0][n][e] + s[1][n][e];
                at[(n * 8 + e) * ss_stride + 8] = s[0][n][e + 2] + s[1][n][e + 2];
              }
            }
          }
        }
      }
      __syncwarp();
      if (lane == 0) tc::mbar_arrive(&k_empty[slot]);
      if (++slot == p.slots) {
        slot = 0;
        phase ^= 1;
      }
      compute_sync();
    }
    compute_sync();
    compute_sync();
  } else if (group == 1) {
    // ---- mixing and softmax: two heads a warp at a time, a key a lane (two with 64 keys a tile)
    compute_sync();
    compute_sync();
    const int j0 = WIDE || lane < bn ? lane : 0;
    for (int index = 0; index < count; ++index) {
      const int key0 = walk.tile(begin + index) * bn;
      const float* s_in = ss + (index & 1) * ss_elems;
      __nv_bfloat16* p_out = ps + (index & 1) * ps_elems + lane;
      float* f_out = corr + (index & 1) * (H + 16);
      const bool ok0 = (WIDE || lane < bn) && !walk.dead(key0 + lane), ok1 = WIDE && !walk.dead(key0 + lane + 32);
      if (!WIDE && bn == 16) {  // sixteen keys: each half of the warp takes one of the two heads
        const bool ok = !walk.dead(key0 + (lane & 15));
        for (int h0 = member; h0 < H; h0 += 2 * GROUP) {
          const bool upper = lane >= 16, used = !upper || h0 + GROUP < H;
          const int h = upper && used ? h0 + GROUP : h0;
          const float* column = s_in + (lane & 15);
          float x = 0.f;
          if (p.talk) {
            const float* t = talk + h * H;
            int g = 0;
            if ((H & 3) == 0) {
#pragma unroll 4
              for (; g < H; g += 4, column += 4 * ss_stride) {
                const float4 w = *reinterpret_cast<const float4*>(t + g);
                x = fmaf(w.x, column[0], x);
                x = fmaf(w.y, column[ss_stride], x);
                x = fmaf(w.z, column[2 * ss_stride], x);
                x = fmaf(w.w, column[3 * ss_stride], x);
              }
            }
            for (; g < H; ++g, column += ss_stride) x = fmaf(t[g], column[0], x);
          } else {
            x = column[h * ss_stride];
          }
          x = ok ? x * p.scale_log2 : -INFINITY;
          const float m_old = m_run[h];
          float m_new = x;
#pragma unroll
          for (int o = 8; o > 0; o >>= 1) m_new = fmaxf(m_new, __shfl_xor_sync(0xffffffffu, m_new, o));
          m_new = fmaxf(m_new, m_old);
          const float a = fast_exp2(x - m_new), factor = fast_exp2(m_old - m_new);
          p_out[h * ps_stride - lane + (lane & 15)] = __float2bfloat16_rn(a);  // (an unused upper half repeats the lower one)
          float sum = a;
#pragma unroll
          for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
          const float l = l_run[h] * factor + sum;
          __syncwarp();
          if ((lane & 15) == 0 && used) {
            m_run[h] = m_new;
            l_run[h] = l;
            f_out[h] = factor;
          }
          __syncwarp();
        }
        compute_sync();
        continue;
      }
      for (int h0 = member; h0 < H; h0 += 2 * GROUP) {
        const int h1 = h0 + GROUP < H ? h0 + GROUP : h0;  // (without a second head: the first one twice, stored once)
        float s[2][2] = {{0.f, 0.f}, {0.f, 0.f}};
        const float* column = s_in + j0;
        if (p.talk) {
          const float *t0 = talk + h0 * H, *t1 = talk + h1 * H;
          int g = 0;
          if ((H & 3) == 0) {
#pragma unroll 4
            for (; g < H; g += 4) {
              const float4 f0 = *reinterpret_cast<const float4*>(t0 + g), f1 = *reinterpret_cast<const float4*>(t1 + g);
              const float w0[4] = {f0.x, f0.y, f0.z, f0.w}, w1[4] = {f1.x, f1.y, f1.z, f1.w};
#pragma unroll
              for (int j = 0; j < 4; ++j) {
                const float a = column[j * ss_stride];
                s[0][0] = fmaf(w0[j], a, s[0][0]);
                s[1][0] = fmaf(w1[j], a, s[1][0]);
                if constexpr (WIDE) {
                  const float b = column[j * ss_stride + 32];
                  s[0][1] = fmaf(w0[j], b, s[0][1]);
                  s[1][1] = fmaf(w1[j], b, s[1][1]);
                }
              }
              column += 4 * ss_stride;
            }
          }
          for (; g < H; ++g, column += ss_stride) {
            const float a = column[0];
            s[0][0] = fmaf(t0[g], a, s[0][0]);
            s[1][0] = fmaf(t1[g], a, s[1][0]);
            if constexpr (WIDE) {
              s[0][1] = fmaf(t0[g], column[32], s[0][1]);
              s[1][1] = fmaf(t1[g], column[32], s[1][1]);
            }
          }
        } else {
          s[0][0] = column[h0 * ss_stride];
          s[1][0] = column[h1 * ss_stride];
          if constexpr (WIDE) {
            s[0][1] = column[h0 * ss_stride + 32];
            s[1][1] = column[h1 * ss_stride + 32];
          }
        }
        const float m_old[2] = {m_run[h0], m_run[h1]};
        float m_new[2], f[2], sum[2];
#pragma unroll
        for (int w = 0; w < 2; ++w) {
          s[w][0] = ok0 ? s[w][0] * p.scale_log2 : -INFINITY;
          s[w][1] = ok1 ? s[w][1] * p.scale_log2 : -INFINITY;
          m_new[w] = WIDE ? fmaxf(s[w][0], s[w][1]) : s[w][0];
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
          for (int w = 0; w < 2; ++w) m_new[w] = fmaxf(m_new[w], __shfl_xor_sync(0xffffffffu, m_new[w], o));
#pragma unroll
        for (int w = 0; w < 2; ++w) {
          m_new[w] = fmaxf(m_new[w], m_old[w]);  // (every tile of the walk holds a key the query sees: finite)
          const float a = fast_exp2(s[w][0] - m_new[w]), b = WIDE ? fast_exp2(s[w][1] - m_new[w]) : 0.f;
          f[w] = fast_exp2(m_old[w] - m_new[w]);
          sum[w] = WIDE ? a + b : a;
          __nv_bfloat16* at = p_out + (w ? h1 : h0) * ps_stride;
          if (WIDE || lane < bn) at[0] = __float2bfloat16_rn(a);
          if constexpr (WIDE) at[32] = __float2bfloat16_rn(b);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
          for (int w = 0; w < 2; ++w) sum[w] += __shfl_xor_sync(0xffffffffu, sum[w], o);
        if (lane == 0) {
          const float l0 = l_run[h0] * f[0] + sum[0], l1 = l_run[h1] * f[1] + sum[1];
          m_run[h0] = m_new[0];
          l_run[h0] = l0;
          f_out[h0] = f[0];
          m_run[h1] = m_new[1];
          l_run[h1] = l1;
          f_out[h1] = f[1];
        }
        __syncwarp();
      }
      compute_sync();
    }
    compute_sync();
  } else {
    // ---- values: O^T of 16 entries x the heads of one KV head a unit
    float acc[MAXU][NT][4];
    int unit_at[MAXU], unit_head[MAXU];  // this lane's offset in a slot, first head of the group (-1: no unit)
#pragma unroll
    for (int u = 0; u < MAXU; ++u) {
      const int unit = member + u * GROUP, c = unit / blocks, chunk = (unit - c * blocks) * 2 + ((lane >> 3) & 1);
      unit_head[u] = unit < units ? c * gs : -1;
      unit_at[u] = (chunk >> 3) * slab_elems + c * box * 64 + lane_row(lane >> 4) + (((chunk & 7) ^ (lane & 7)) << 3);
#pragma unroll
      for (int n = 0; n < NT; ++n) acc[u][n][0] = acc[u][n][1] = acc[u][n][2] = acc[u][n][3] = 0.f;
    }
    compute_sync();
    compute_sync();
    compute_sync();
    for (int index = 0; index < count; ++index) {
      const __nv_bfloat16* p_in = ps + (index & 1) * ps_elems;
      const float* f_in = corr + (index & 1) * (H + 16);
      __nv_bfloat16* values = v_ring + slot * slot_elems;
      tc::mbar_wait(&v_full[slot], phase, abort_flag, &g_error_word, 3);
      if (walk.edge(begin + index)) {
        // value rows no query sees hold whatever their page held before: weight 0, but 0 x NaN is NaN
        const int key0 = walk.tile(begin + index) * bn;
        for (int i = threadIdx.x - 2 * GROUP * 32; i < bn * G * (P / 8); i += GROUP * 32) {
          const int chunk = i % (P / 8), rest = i / (P / 8), c = rest % G, key = rest / G;
          if (walk.dead(key0 + key))
            *reinterpret_cast<uint4*>(values + (chunk >> 3) * slab_elems +
                                      (((key >> p.box_shift) * G + c) * box + (key & (box - 1))) * 64 +
                                      (((chunk & 7) ^ (key & 7)) << 3)) = make_uint4(0u, 0u, 0u, 0u);
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // a later copy may refill the slot
        asm volatile("bar.sync 2, %0;" ::"n"(GROUP * 32) : "memory");  // (the value warps)
      }
#pragma unroll
      for (int u = 0; u < MAXU; ++u) {
        if (unit_head[u] < 0) break;
        const float* factor = f_in + unit_head[u] + (lane & 3) * 2;
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          acc[u][n][0] *= factor[n * 8];
          acc[u][n][1] *= factor[n * 8 + 1];
          acc[u][n][2] *= factor[n * 8];
          acc[u][n][3] *= factor[n * 8 + 1];
        }
        const __nv_bfloat16* block = values + unit_at[u];
        const __nv_bfloat16* prow = p_in + (unit_head[u] + (lane >> 2)) * ps_stride + (lane & 3) * 2;
#pragma unroll
        for (int kb = 0; kb < (WIDE ? 4 : 2); ++kb) {
          if (!WIDE && kb >= key_blocks) break;
          unsigned a[4];
          ldmatrix_x4_trans(a, block + kb * block_step);
#pragma unroll
          for (int n = 0; n < NT; ++n) {
            const __nv_bfloat16* at = prow + n * 8 * ps_stride + kb * 16;
            mma_16816(acc[u][n], a, *reinterpret_cast<const unsigned*>(at), *reinterpret_cast<const unsigned*>(at + 8));
          }
        }
      }
      __syncwarp();
      if (lane == 0) tc::mbar_arrive(&v_empty[slot]);
      if (++slot == p.slots) {
        slot = 0;
        phase ^= 1;
      }
      compute_sync();
    }
    // the heads' outputs to shared memory, over the rings (every copy into them has landed and been read)
    float* os = reinterpret_cast<float*>(base);  // [H][P + 4]
#pragma unroll
    for (int u = 0; u < MAXU; ++u) {
      const int unit = member + u * GROUP, entry = (unit % blocks) * 16;
      if (unit_head[u] < 0) break;
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int head = n * 8 + (lane & 3) * 2 + (e & 1);
          if (head < gs) os[(unit_head[u] + head) * (P + 4) + entry + (lane >> 2) + (e >> 1) * 8] = acc[u][n][e];
        }
    }
  }
  // ---- then to memory in whole rows
  constexpr int OS = P + 4;
  const float* os = reinterpret_cast<const float*>(base);
  compute_sync();
  __nv_bfloat16* out = p.out + (size_t)token * p.out_stride;
  if (my_splits == 1) {
    for (int i = threadIdx.x; i < H * p.v_cols; i += COMPUTE) {
      const int h = i / p.v_cols, c = i - h * p.v_cols;
      out[i] = __float2bfloat16_rn(os[h * OS + c] / l_run[h]);
    }
    return;
  }
  const size_t item = (size_t)tile_index * p.splits + split;
  const int quads = blocks * 4;  // 16-byte pieces of a head's row that hold anything
  for (int i = threadIdx.x; i < H * quads; i += COMPUTE) {
    const int h = i / quads, c = (i - h * quads) * 4;
    *reinterpret_cast<float4*>(p.part_acc + (item * H + h) * P + c) = *reinterpret_cast<const float4*>(os + h * OS + c);
  }
  for (int h = threadIdx.x; h < H; h += COMPUTE)
    *reinterpret_cast<float2*>(p.part_ml + (item * H + h) * 2) = make_float2(m_run[h], l_run[h]);
  // ---- the share that is written last merges all of them
  __shared__ int last_to_arrive;
  compute_sync();
  if (threadIdx.x == 0) {
    int ticket;  // releases this CTA's partial results; the last one acquires the others'
    asm volatile("atom.add.acq_rel.gpu.global.s32 %0, [%1], 1;" : "=r"(ticket) : "l"(p.arrivals + tile_index) : "memory");
    last_to_arrive = ticket == my_splits - 1;
    if (last_to_arrive) p.arrivals[tile_index] = 0;  // zero again for the next launch
  }
  compute_sync();
  if (!last_to_arrive) return;
  const size_t first = (size_t)tile_index * p.splits;
  for (int i = threadIdx.x; i < H * quads; i += COMPUTE) {
    const int h = i / quads, c = (i - h * quads) * 4;
    const float2* ml = reinterpret_cast<const float2*>(p.part_ml) + first * H + h;
    const float4* src = reinterpret_cast<const float4*>(p.part_acc + (first * H + h) * P + c);
    float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
    float m_ref = -INFINITY, l = 0.f;
    constexpr int BATCH = 8;  // shares whose loads are in flight at once
    for (int s = 0; s < my_splits; s += BATCH) {
      float4 v[BATCH];
      float2 w[BATCH];
#pragma unroll
      for (int j = 0; j < BATCH; ++j) {
        const bool used = s + j < my_splits;
        w[j] = used ? __ldcg(ml + (size_t)(s + j) * H) : make_float2(-INFINITY, 0.f);
        v[j] = used ? __ldcg(src + (size_t)(s + j) * H * (P / 4)) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
      float m_new = m_ref;
#pragma unroll
      for (int j = 0; j < BATCH; ++j) m_new = fmaxf(m_new, w[j].x);
      const float m_use = m_new == -INFINITY ? 0.f : m_new;
      const float f0 = exp2f(m_ref - m_use);
      sum.x *= f0; sum.y *= f0; sum.z *= f0; sum.w *= f0;
      l *= f0;
      m_ref = m_new;
#pragma unroll
      for (int j = 0; j < BATCH; ++j) {
        const float f = exp2f(w[j].x - m_use);  // 0 for the unused ones
        l = fmaf(w[j].y, f, l);
        sum.x = fmaf(v[j].x, f, sum.x);
        sum.y = fmaf(v[j].y, f, sum.y);
        sum.z = fmaf(v[j].z, f, sum.z);
        sum.w = fmaf(v[j].w, f, sum.w);
      }
    }
    const float inv = 1.f / l, r[4] = {sum.x * inv, sum.y * inv, sum.z * inv, sum.w * inv};
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (c + e < p.v_cols) out[h * p.v_cols + c + e] = __float2bfloat16_rn(r[e]);
  }
}

// ------------------------------------------------------------------ host side
struct MapKey {
  const void* base;
  uint64_t rows;
  uint32_t size, page, box, heads;
  bool operator==(const MapKey& o) const {
    return base == o.base && rows == o.rows && size == o.size && page == o.page && box == o.box && heads == o.heads;
  }
};
struct MapKeyHash {
  size_t operator()(const MapKey& k) const {
    size_t h = reinterpret_cast<size_t>(k.base);
    for (uint64_t x : {k.rows, (uint64_t)k.size, (uint64_t)k.page, (uint64_t)k.box, (uint64_t)k.heads}) h = h * 1000003u ^ x;
    return h;
  }
};

// The cache layer as [rows = pages x planes x KV heads][page_size][P]: boxes of KV heads x ``box`` positions x 64 entries.
bool cached_map(CUtensorMap* out, const MapKey& key) {
  static std::unordered_map<MapKey, CUtensorMap, MapKeyHash> cache;
  static std::mutex lock;
  std::lock_guard<std::mutex> guard(lock);
  auto it = cache.find(key);
  if (it == cache.end()) {
    tc_host::EncodeTiledFn fn = tc_host::encode_fn();
    if (!fn || (reinterpret_cast<uintptr_t>(key.base) & 15)) return false;
    cuuint64_t dims[3] = {key.size, key.page, key.rows};
    cuuint64_t strides[2] = {(cuuint64_t)key.size * 2, (cuuint64_t)key.page * key.size * 2};
    cuuint32_t box[3] = {64, key.box, key.heads};
    cuuint32_t elem[3] = {1, 1, 1};
    CUtensorMap map;
    if (fn(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(key.base), dims, strides, box, elem,
           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
      return false;
    if (cache.size() > 1024) cache.clear();
    it = cache.emplace(key, map).first;
  }
  *out = it->second;
  return true;
}

int keys_a_tile(int G, int P) {
  int bn = 64;
  while (bn > 16 && 2 * G * bn * P * 2 > TILE_LIMIT) bn >>= 1;
  return bn;
}

size_t smem_bytes(int H, int G, int P, int bn, bool talk, int slots) {
  size_t bytes = (size_t)slots * 2 * G * bn * P * 2;
  const int row = bn > 32 ? 64 : 32;
  bytes += 2 * ((size_t)(H + 16) * (row + 8) * 2 + (size_t)H * (row + 4) * 4);
  bytes += (talk ? (size_t)H * H * 4 : 0) + (size_t)(4 * H + 32) * 4;
  return bytes + 1024 + 8 + 4 * MAX_SLOTS * 8 + 64;
}
int slots_for(int H, int G, int P, int bn) {
  for (int slots = MAX_SLOTS; slots >= 2; --slots)
    if (smem_bytes(H, G, P, bn, true, slots) <= SMEM_LIMIT - 1024 &&
        (size_t)H * (P + 4) * 4 <= (size_t)slots * 2 * G * bn * P * 2)  // the heads' outputs lie over the rings at the end
      return slots;
  return 0;
}

int log2_exact(int v) {
  for (int b = 0; b < 12; ++b)
    if ((1 << b) == v) return b;
  return -1;
}

template <int P, int NT, int MAXU, bool WIDE>
int launch(const CUtensorMap& map, const Params& p, int tiles, size_t smem, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    cudaError_t err = cudaFuncSetAttribute(attention_mixed_decode_kernel<P, NT, MAXU, WIDE>,
                                           cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_LIMIT - 1024);
    if (err != cudaSuccess) return (int)err;
    configured = true;
  }
  tl::launch_kernel(attention_mixed_decode_kernel<P, NT, MAXU, WIDE>, dim3(tiles, p.splits), THREADS, smem, stream, map, p);
  return TL_LAUNCH_CHECK();
}

int units_each(int G, int v_cols) { return (G * ((v_cols + 15) / 16) + GROUP - 1) / GROUP; }

// (tiles of 64 keys mean G P <= 256: at most two units a warp)
template <int P, int NT>
int launch_units(const CUtensorMap& map, const Params& p, int tiles, size_t smem, cudaStream_t stream) {
  const int each = units_each(p.G, p.v_cols);
  if (p.bn == 64) return each <= 2 ? launch<P, NT, 2, true>(map, p, tiles, smem, stream) : TL_ERR_UNSUPPORTED;
  if (each <= 4) return launch<P, NT, 4, false>(map, p, tiles, smem, stream);
  if constexpr (NT == 1)
    if (each <= 8) return launch<P, NT, 8, false>(map, p, tiles, smem, stream);
  return TL_ERR_UNSUPPORTED;
}

}  // namespace

TL_DEBUG_READER(tl_attention_mixed_decode_debug_error)

extern "C" {

int tl_attention_mixed_decode_error() {
  int value = 0, zero = 0;
  if (cudaMemcpyFromSymbol(&value, g_error_word, sizeof(int)) != cudaSuccess) return -1;
  if (value) cudaMemcpyToSymbol(g_error_word, &zero, sizeof(int));
  return value;
}

// Keys a tile holds for these sizes, or 0 where the kernel does not take them.
int tl_attention_mixed_decode_tile(int H, int G, int P, int page_size, int v_cols) {
  if ((P != 64 && P != 128) || G <= 0 || H <= 0 || H % G || H > MAX_HEADS || H / G > 16 || v_cols <= 0 || v_cols > P) return 0;
  if (page_size < 8 || page_size > 4096 || log2_exact(page_size) < 0) return 0;
  if (units_each(G, v_cols) > (H / G <= 8 ? 8 : 4)) return 0;
  const int bn = keys_a_tile(G, P);
  return slots_for(H, G, P, bn) ? bn : 0;
}

// Bytes of float32 workspace for ``splits`` shares of ``tiles`` requests.
long long tl_attention_mixed_decode_workspace(int tiles, int H, int P, int splits) {
  return splits > 1 ? (long long)tiles * splits * H * (P + 2) * 4 : 0;
}

// q [tokens][nh][p_size] bf16 rows (q_stride elements apart); pages [num_pages][2][nkv][page_size][p_size] bf16; tile_req:
// the requests that bring ONE token (null: request i for every tile i); arrivals [tiles]: zero before and after.
// talk [nh][nh] float32 or null.  out [tokens][out_stride]: v_cols entries a head.
int tl_attention_mixed_decode(const void* q, long long q_stride, const void* pages, long long num_pages,
                              const int* block_table, int table_width, const int* req_indptr, const int* kv_before,
                              const int* tile_req, int tiles, void* out, long long out_stride, int nh, int nkv, int p_size,
                              int page_size, int window, int keep, int v_cols, float scale, const float* talk, int splits,
                              void* workspace, long long workspace_bytes, int* arrivals, cudaStream_t stream) {
  if (tiles <= 0) return 0;
  const int bn = tl_attention_mixed_decode_tile(nh, nkv, p_size, page_size, v_cols);
  if (!bn || q_stride % 8 || (reinterpret_cast<uintptr_t>(q) & 15) || keep < 0 || splits < 1 || splits > 65535)
    return TL_ERR_UNSUPPORTED;
  if (splits > 1 && (!arrivals || workspace_bytes < tl_attention_mixed_decode_workspace(tiles, nh, p_size, splits)))
    return TL_ERR_UNSUPPORTED;
  const int box = page_size < 16 ? page_size : 16;
  CUtensorMap map;
  if (!cached_map(&map, MapKey{pages, (uint64_t)num_pages * 2 * nkv, (uint32_t)p_size, (uint32_t)page_size, (uint32_t)box,
                               (uint32_t)nkv}))
    return TL_ERR_UNSUPPORTED;
  Params p;
  memset(&p, 0, sizeof(p));
  p.q = (const __nv_bfloat16*)q;
  p.q_stride = q_stride;
  p.block_table = block_table;
  p.table_width = table_width;
  p.req_indptr = req_indptr;
  p.kv_before = kv_before;
  p.tile_req = tile_req;
  p.out = (__nv_bfloat16*)out;
  p.out_stride = out_stride;
  p.part_acc = (float*)workspace;
  p.part_ml = p.part_acc + (size_t)tiles * splits * nh * p_size;
  p.arrivals = arrivals;
  p.H = nh;
  p.G = nkv;
  p.page_shift = log2_exact(page_size);
  p.window = window;
  p.keep = window > 0 ? keep : 0;
  p.v_cols = v_cols;
  p.splits = splits;
  p.bn = bn;
  p.box_shift = log2_exact(box);
  p.talk = talk;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.num_pages = (int)num_pages;
  p.slots = slots_for(nh, nkv, p_size, bn);
  const size_t smem = smem_bytes(nh, nkv, p_size, bn, talk != nullptr, p.slots);
  const bool one = nh / nkv <= 8;
  if (p_size == 128)
    return one ? launch_units<128, 1>(map, p, tiles, smem, stream) : launch_units<128, 2>(map, p, tiles, smem, stream);
  return one ? launch_units<64, 1>(map, p, tiles, smem, stream) : launch_units<64, 2>(map, p, tiles, smem, stream);
}

}  // extern "C"
