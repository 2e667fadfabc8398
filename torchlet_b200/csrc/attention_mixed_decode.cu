// Paged attention of SINGLE TOKENS, bfloat16 on the tensor cores, for scores that are mixed across the heads before the
// softmax (s_h <- sum_g T[h, g] s_g) and a sliding window that may keep the sequence's first tokens.  Head rows of P = 64 or
// 128 entries, up to 16 query heads a KV head.
//
// Mixing needs the scores of ALL heads with a key at once, so one CTA takes all heads of a request over a share of its key
// tiles (blockIdx.y; the last CTA of a request to finish merges the shares), and every key and value row is read once:
//
//   keys and values  tiles of BN = 16, 32 or 64 absolute positions (as many as keep a stage at 64 KB or less), K and V of all
//                    KV heads, by TMA: 3-D boxes of 64 entries x positions of a page x KV heads (128-byte swizzle), three
//                    stages; first the tiles of kept positions that lie wholly before the window, then the window's
//   scores           S^T [keys x heads of a group] = K Q^T a KV head, mma.sync m16n8k16 with the keys as rows: a group of up
//                    to eight heads fills one column tile; the float32 scores go to shared memory
//   softmax          one warp a head: the mixed score of a key a lane, float32, running max and sum
//   values           O^T [entries x heads of a group] += V^T P^T, 16 entries of one KV head a warp and unit, accumulators in
//                    registers for the whole walk
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

constexpr int WARPS = 8;
constexpr int THREADS = WARPS * 32;
constexpr int STAGES = 3;
constexpr int MAX_HEADS = 64;
constexpr int STAGE_LIMIT = 64 * 1024;
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

// Where a row of a stage lies: plane (0 K, 1 V), KV head, key within the tile, 8-entry chunk.
template <int P> __device__ __forceinline__ __nv_bfloat16* kv_at(__nv_bfloat16* stage, const Params& p, int plane, int c, int key, int chunk) {
  const int slab_elems = p.G * p.bn * 64, box = 1 << p.box_shift;
  const int row = ((key >> p.box_shift) * p.G + c) * box + (key & (box - 1));
  return stage + (plane * (P / 64) + (chunk >> 3)) * slab_elems + row * 64 + (((chunk & 7) ^ (key & 7)) << 3);
}

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
  // tiles a CTA takes and how many CTAs that makes, out of the ``splits`` the grid holds: no share below 64 keys
  __device__ __forceinline__ int share(int splits) const { return max(max(1, 64 / bn), (count + splits - 1) / splits); }
};

// NT: column tiles of eight heads a group; MAXU: units of 16 value entries a warp accumulates.
template <int P, int NT, int MAXU>
__global__ void __launch_bounds__(THREADS, 1)
attention_mixed_decode_kernel(const __grid_constant__ CUtensorMap map_kv, const Params p) {
  constexpr int SLABS = P / 64, QS = P + 8;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int bn = p.bn, H = p.H, G = p.G, gs = H / G;
  const int stage_elems = 2 * G * bn * P;
  __nv_bfloat16* stages = reinterpret_cast<__nv_bfloat16*>(base);
  __nv_bfloat16* qs = stages + STAGES * stage_elems;                    // [H + 16][QS]
  const int ps_stride = bn + 8, ss_stride = bn + 4;
  __nv_bfloat16* ps = qs + (H + 16) * QS;                               // [H + 16][bn + 8]
  float* ss = reinterpret_cast<float*>(ps + (H + 16) * ps_stride);      // [H][bn + 4]
  float* talk = ss + H * ss_stride;                                     // [H][H]
  float* m_run = talk + (p.talk ? H * H : 0);                           // [H]
  float* l_run = m_run + H;                                             // [H]
  float* corr = l_run + H;                                              // [H + 16]
  uint64_t* full = reinterpret_cast<uint64_t*>((reinterpret_cast<uintptr_t>(corr + H + 16) + 7) & ~(uintptr_t)7);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(full + STAGES);

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
    for (int i = 0; i < STAGES; ++i) tc::mbar_init(&full[i], 1);
    *abort_flag = 0;
    tc::mbar_fence_init();
    tc::prefetch_tensormap(&map_kv);
  }
  __syncthreads();

  // requests the tile ``index`` (of this CTA's) into its stage: warp 0, one lane a box
  const int box = 1 << p.box_shift, boxes_per_tile = bn >> p.box_shift;
  auto request = [&](int index) {
    const int stage = index % STAGES, key0 = walk.tile(begin + index) * bn;
    if (lane == 0) tc::mbar_expect_tx(&full[stage], (uint32_t)stage_elems * 2);
    __syncwarp();
    for (int b = lane; b < 2 * SLABS * boxes_per_tile; b += 32) {
      const int part = b % boxes_per_tile, slab = (b / boxes_per_tile) % SLABS, plane = b / (boxes_per_tile * SLABS);
      const int key = key0 + part * box, entry = key >> p.page_shift;
      int page = (entry < p.table_width && key <= walk.hi) ? table[entry] : 0;  // beyond the last key: page 0, which is always there
      if (!TL_DEBUG_OK(page >= 0 && page < p.num_pages, TL_DEBUG_PAGE, page)) page = 0;
      __nv_bfloat16* dst = stages + stage * stage_elems + (plane * SLABS + slab) * (G * bn * 64) + part * (G * box * 64);
      tc::tma_load_3d(dst, &map_kv, &full[stage], slab * 64, key & ((1 << p.page_shift) - 1), (page * 2 + plane) * G);
    }
  };
  // tiles that earlier steps wrote may be requested before the wait on the preceding kernel
  int issued = 0;
  if (warp == 0)
    while (issued < min(STAGES, count) && walk.tile(begin + issued) * bn + bn - 1 < before) request(issued++);
  pdl_wait();
  pdl_launch_dependents();
  if (warp == 0)
    while (issued < min(STAGES, count)) request(issued++);

  for (int i = threadIdx.x; i < H * (P / 8); i += THREADS) {
    const int h = i / (P / 8), c = i % (P / 8);
    *reinterpret_cast<uint4*>(qs + h * QS + c * 8) =
        *reinterpret_cast<const uint4*>(p.q + (size_t)token * p.q_stride + (size_t)h * P + c * 8);
  }
  // the rows behind the last head fill a group's column tile: their columns are computed and never used
  for (int i = threadIdx.x; i < 16 * QS; i += THREADS) qs[H * QS + i] = __float2bfloat16_rn(0.f);
  for (int i = threadIdx.x; i < 16 * ps_stride; i += THREADS) ps[H * ps_stride + i] = __float2bfloat16_rn(0.f);
  if (p.talk)
    for (int i = threadIdx.x; i < H * H; i += THREADS) talk[i] = p.talk[i];
  for (int i = threadIdx.x; i < H + 16; i += THREADS) {
    if (i < H) {
      m_run[i] = -INFINITY;
      l_run[i] = 0.f;
    }
    corr[i] = 0.f;
  }
  __syncthreads();

  const int blocks = (p.v_cols + 15) / 16;  // units of 16 value entries a KV head
  const int units = G * blocks;
  float acc[MAXU][NT][4];
#pragma unroll
  for (int u = 0; u < MAXU; ++u)
#pragma unroll
    for (int n = 0; n < NT; ++n) acc[u][n][0] = acc[u][n][1] = acc[u][n][2] = acc[u][n][3] = 0.f;

  const int key_blocks = bn >> 4;
  for (int index = 0; index < count; ++index) {
    const int stage = index % STAGES, key0 = walk.tile(begin + index) * bn;
    __nv_bfloat16* kv = stages + stage * stage_elems;
    tc::mbar_wait(&full[stage], (index / STAGES) & 1, abort_flag, &g_error_word, 1);
    if (walk.edge(begin + index)) {
      // value rows no query sees hold whatever their page held before: weight 0, but 0 x NaN is NaN
      for (int i = threadIdx.x; i < bn * G * (P / 8); i += THREADS) {
        const int chunk = i % (P / 8), rest = i / (P / 8), c = rest % G, key = rest / G;
        if (walk.dead(key0 + key)) *reinterpret_cast<uint4*>(kv_at<P>(kv, p, 1, c, key, chunk)) = make_uint4(0u, 0u, 0u, 0u);
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // a later copy may refill the stage
    }
    // ---- scores: S^T of 16 keys x the heads of one group a unit
    for (int u = warp; u < G * key_blocks; u += WARPS) {
      const int c = u % G, kb = u / G;
      float s[NT][4];
#pragma unroll
      for (int n = 0; n < NT; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
      const int key = kb * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
      const __nv_bfloat16* qrow = qs + (c * gs + (lane >> 2)) * QS + (lane & 3) * 2;
#pragma unroll
      for (int k = 0; k < P / 16; ++k) {
        unsigned a[4];
        ldmatrix_x4(a, kv_at<P>(kv, p, 0, c, key, 2 * k + (lane >> 4)));
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const __nv_bfloat16* at = qrow + n * 8 * QS + k * 16;
          mma_16816(s[n], a, *reinterpret_cast<const unsigned*>(at), *reinterpret_cast<const unsigned*>(at + 8));
        }
      }
#pragma unroll
      for (int n = 0; n < NT; ++n) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int head = n * 8 + (lane & 3) * 2 + (e & 1);
          if (head < gs) ss[(c * gs + head) * ss_stride + kb * 16 + (lane >> 2) + (e >> 1) * 8] = s[n][e];
        }
      }
    }
    __syncthreads();  // scores are here, and every warp is done with the tile before: its stage may be refilled
    if (warp == 0 && index > 0 && index + STAGES - 1 < count) request(index + STAGES - 1);
    // ---- mixing and softmax: two heads a warp at a time, a key a lane (two with 64 keys a tile)
    for (int h0 = warp; h0 < H; h0 += 2 * WARPS) {
      const int h1 = h0 + WARPS;
      const bool two = h1 < H;
      float s0[2] = {0.f, 0.f}, s1[2] = {0.f, 0.f};
      const int j0 = lane < bn ? lane : 0, j1 = bn > 32 ? lane + 32 : j0;
      if (p.talk) {
        const float *t0 = talk + h0 * H, *t1 = talk + (two ? h1 : h0) * H;
#pragma unroll 4
        for (int g = 0; g < H; ++g) {
          const float a = ss[g * ss_stride + j0], b = ss[g * ss_stride + j1];
          s0[0] = fmaf(t0[g], a, s0[0]);
          s0[1] = fmaf(t0[g], b, s0[1]);
          s1[0] = fmaf(t1[g], a, s1[0]);
          s1[1] = fmaf(t1[g], b, s1[1]);
        }
      } else {
        s0[0] = ss[h0 * ss_stride + j0];
        s0[1] = ss[h0 * ss_stride + j1];
        s1[0] = ss[(two ? h1 : h0) * ss_stride + j0];
        s1[1] = ss[(two ? h1 : h0) * ss_stride + j1];
      }
      const bool ok0 = lane < bn && !walk.dead(key0 + lane), ok1 = bn > 32 && !walk.dead(key0 + lane + 32);
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        if (w == 1 && !two) break;
        const int h = w == 0 ? h0 : h1;
        const float a = ok0 ? (w == 0 ? s0[0] : s1[0]) * p.scale_log2 : -INFINITY;
        const float b = ok1 ? (w == 0 ? s0[1] : s1[1]) * p.scale_log2 : -INFINITY;
        const float m_old = m_run[h], m_new = fmaxf(m_old, warp_max(fmaxf(a, b)));
        const float m_use = m_new == -INFINITY ? 0.f : m_new;
        const float pa = exp2f(a - m_use), pb = exp2f(b - m_use), f = exp2f(m_old - m_use);
        const float sum = warp_sum(pa + pb);
        if (lane < bn) ps[h * ps_stride + lane] = __float2bfloat16_rn(pa);
        if (bn > 32) ps[h * ps_stride + lane + 32] = __float2bfloat16_rn(pb);
        __syncwarp();
        if (lane == 0) {
          m_run[h] = m_new;
          l_run[h] = l_run[h] * f + sum;
          corr[h] = f;
        }
      }
    }
    __syncthreads();
    // ---- values: O^T of 16 entries x the heads of one group a unit
#pragma unroll
    for (int i = 0; i < MAXU; ++i) {
      const int u = warp + i * WARPS;
      if (u < units) {
        const int c = u / blocks, db = u % blocks;
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const float f0 = corr[c * gs + n * 8 + (lane & 3) * 2], f1 = corr[c * gs + n * 8 + (lane & 3) * 2 + 1];
          acc[i][n][0] *= f0;
          acc[i][n][1] *= f1;
          acc[i][n][2] *= f0;
          acc[i][n][3] *= f1;
        }
        for (int kb = 0; kb < key_blocks; ++kb) {
          unsigned a[4];
          ldmatrix_x4_trans(a, kv_at<P>(kv, p, 1, c, kb * 16 + (lane & 7) + (lane >> 4) * 8, db * 2 + ((lane >> 3) & 1)));
          const __nv_bfloat16* prow = ps + (c * gs + (lane >> 2)) * ps_stride + kb * 16 + (lane & 3) * 2;
#pragma unroll
          for (int n = 0; n < NT; ++n) {
            const __nv_bfloat16* at = prow + n * 8 * ps_stride;
            mma_16816(acc[i][n], a, *reinterpret_cast<const unsigned*>(at), *reinterpret_cast<const unsigned*>(at + 8));
          }
        }
      }
    }
  }
  __syncthreads();
  // ---- the heads' outputs to shared memory (over the stages), then to memory in whole rows
  constexpr int OS = P + 4;
  float* os = reinterpret_cast<float*>(stages);  // [H][OS]
#pragma unroll
  for (int i = 0; i < MAXU; ++i) {
    const int u = warp + i * WARPS;
    if (u < units) {
      const int c = u / blocks, db = u % blocks;
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int head = n * 8 + (lane & 3) * 2 + (e & 1);
          if (head < gs) os[(c * gs + head) * OS + db * 16 + (lane >> 2) + (e >> 1) * 8] = acc[i][n][e];
        }
    }
  }
  __syncthreads();
  __nv_bfloat16* out = p.out + (size_t)token * p.out_stride;
  if (my_splits == 1) {
    for (int i = threadIdx.x; i < H * p.v_cols; i += THREADS) {
      const int h = i / p.v_cols, c = i - h * p.v_cols;
      out[i] = __float2bfloat16_rn(os[h * OS + c] / l_run[h]);
    }
    return;
  }
  const size_t item = (size_t)tile_index * p.splits + split;
  const int quads = blocks * 4;  // 16-byte pieces of a head's row that hold anything
  for (int i = threadIdx.x; i < H * quads; i += THREADS) {
    const int h = i / quads, c = (i - h * quads) * 4;
    *reinterpret_cast<float4*>(p.part_acc + (item * H + h) * P + c) = *reinterpret_cast<const float4*>(os + h * OS + c);
  }
  for (int h = threadIdx.x; h < H; h += THREADS)
    *reinterpret_cast<float2*>(p.part_ml + (item * H + h) * 2) = make_float2(m_run[h], l_run[h]);
  // ---- the share that is written last merges all of them
  __shared__ int last_to_arrive;
  __syncthreads();
  if (threadIdx.x == 0) {
    int ticket;  // releases this CTA's partial results; the last one acquires the others'
    asm volatile("atom.add.acq_rel.gpu.global.s32 %0, [%1], 1;" : "=r"(ticket) : "l"(p.arrivals + tile_index) : "memory");
    last_to_arrive = ticket == my_splits - 1;
    if (last_to_arrive) p.arrivals[tile_index] = 0;  // zero again for the next launch
  }
  __syncthreads();
  if (!last_to_arrive) return;
  const size_t first = (size_t)tile_index * p.splits;
  for (int i = threadIdx.x; i < H * quads; i += THREADS) {
    const int h = i / quads, c = (i - h * quads) * 4;
    const float2* ml = reinterpret_cast<const float2*>(p.part_ml) + first * H + h;
    const float4* src = reinterpret_cast<const float4*>(p.part_acc + (first * H + h) * P + c);
    float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
    float m_ref = -INFINITY, l = 0.f;
    for (int s = 0; s < my_splits; s += 8) {  // eight shares' loads in flight
      float4 v[8];
      float2 w[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const bool used = s + j < my_splits;
        w[j] = used ? __ldcg(ml + (size_t)(s + j) * H) : make_float2(-INFINITY, 0.f);
        v[j] = used ? __ldcg(src + (size_t)(s + j) * H * (P / 4)) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
      float m_new = m_ref;
#pragma unroll
      for (int j = 0; j < 8; ++j) m_new = fmaxf(m_new, w[j].x);
      const float m_use = m_new == -INFINITY ? 0.f : m_new;
      const float f0 = exp2f(m_ref - m_use);
      sum.x *= f0; sum.y *= f0; sum.z *= f0; sum.w *= f0;
      l *= f0;
      m_ref = m_new;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
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
  while (bn > 16 && 2 * G * bn * P * 2 > STAGE_LIMIT) bn >>= 1;
  return bn;
}

size_t smem_bytes(int H, int G, int P, int bn, bool talk) {
  size_t bytes = (size_t)STAGES * 2 * G * bn * P * 2;
  bytes += (size_t)(H + 16) * (P + 8) * 2 + (size_t)(H + 16) * (bn + 8) * 2 + (size_t)H * (bn + 4) * 4;
  bytes += (talk ? (size_t)H * H * 4 : 0) + (size_t)(3 * H + 16) * 4;
  return bytes + 1024 + 8 + STAGES * 8 + 64;
}

int log2_exact(int v) {
  for (int b = 0; b < 12; ++b)
    if ((1 << b) == v) return b;
  return -1;
}

template <int P, int NT, int MAXU>
int launch(const CUtensorMap& map, const Params& p, int tiles, size_t smem, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    cudaError_t err = cudaFuncSetAttribute(attention_mixed_decode_kernel<P, NT, MAXU>,
                                           cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_LIMIT - 1024);
    if (err != cudaSuccess) return (int)err;
    configured = true;
  }
  tl::launch_kernel(attention_mixed_decode_kernel<P, NT, MAXU>, dim3(tiles, p.splits), THREADS, smem, stream, map, p);
  return TL_LAUNCH_CHECK();
}

template <int P, int NT>
int launch_units(const CUtensorMap& map, const Params& p, int tiles, size_t smem, cudaStream_t stream) {
  const int each = (p.G * ((p.v_cols + 15) / 16) + WARPS - 1) / WARPS;
  if (each <= 1) return launch<P, NT, 1>(map, p, tiles, smem, stream);
  if (each <= 2) return launch<P, NT, 2>(map, p, tiles, smem, stream);
  if (each <= 4) return launch<P, NT, 4>(map, p, tiles, smem, stream);
  if (each <= 8) return launch<P, NT, 8>(map, p, tiles, smem, stream);
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
  if ((G * ((v_cols + 15) / 16) + WARPS - 1) / WARPS > 8) return 0;
  const int bn = keys_a_tile(G, P);
  if (smem_bytes(H, G, P, bn, true) > SMEM_LIMIT - 1024) return 0;
  if ((size_t)H * (P + 4) * 4 > (size_t)STAGES * 2 * G * bn * P * 2) return 0;
  return bn;
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
  const int box = bn < page_size ? bn : page_size;
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
  const size_t smem = smem_bytes(nh, nkv, p_size, bn, talk != nullptr);
  const bool one = nh / nkv <= 8;
  if (p_size == 128)
    return one ? launch_units<128, 1>(map, p, tiles, smem, stream) : launch_units<128, 2>(map, p, tiles, smem, stream);
  return one ? launch_units<64, 1>(map, p, tiles, smem, stream) : launch_units<64, 2>(map, p, tiles, smem, stream);
}

}  // extern "C"
