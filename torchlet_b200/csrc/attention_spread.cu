// Paged causal attention of PROMPT PORTIONS on the 5th-generation tensor cores (tcgen05), bfloat16, for two options the
// plain prompt kernel (attention_tc.cu) does not have: scores MIXED ACROSS THE HEADS before the softmax, and a sliding
// window beside which the sequence's first ``keep`` tokens stay visible.  Head rows of P = 64 or 128 entries.
//
// Mixed scores are linear in the queries, so the caller spreads each mixed query over all KV heads (qkv_prepare.cu): a
// query row is ``chunks`` = G pieces of P entries, one a KV head, and its score with a token is the sum of the pieces' dot
// products with that token's G keys.  Without mixing ``chunks`` is 1 and the piece belongs to the row's own KV head.
//
// One CTA takes a tile of up to 128 PACKED ROWS of one (request, KV head): the pairs (token of the step, query head of the
// KV head's group), token-major.  It walks over the keys in tiles of 128 absolute positions: first the tiles of kept
// positions that lie wholly before the window, then the window's.
//
//   loader warps    one for K (``chunks`` operand tiles a key tile, one a KV head), one for V: TMA boxes of
//                   page_size x 64 elements through the block table into rings (128-byte swizzle, one lane a box).  The
//                   query pieces are loaded once, by 3-D TMA boxes (64 elements x heads of the group x tokens); where
//                   they do not fit the shared memory they come along with each K tile instead.
//   MMA warp        S_j = sum over the pieces of Q_c K_c^T (accumulated in tensor memory), then O += P_(j-1) V of the
//                   previous key tile (P read from tensor memory).  S has two buffers, so the tensor cores multiply the
//                   next tile's scores while this tile is in its softmax.
//   softmax warps   four, one thread per row: the row of S from tensor memory, mask by position, running max and sum in
//                   float32, P as bfloat16 over the first half of S's columns; O is rescaled in tensor memory when the
//                   row's max has grown by more than 2^8 (behind the P V in flight).
//
// Numerics as in attention_tc.cu: float32 scores, max, sum and accumulator, P rounded to bfloat16 before P V.  Every wait is
// bounded (tcgen05.cuh); one that gives up leaves a code that tl_attention_spread_error() returns.
#include <math.h>
#include <string.h>

#include <mutex>
#include <unordered_map>

#include "common.cuh"
#include "tcgen05.cuh"

namespace {

using namespace tc;

constexpr int ROWS = 128;  // packed rows of a tile (UMMA M)
constexpr int KEYS = 128;  // keys a tile (UMMA N of S, K of P V)
constexpr int THREADS = 224;  // warps 0-3 softmax, 4 MMA, 5 K (and Q) loader, 6 V loader
constexpr int SLAB = ROWS * 128;  // bytes of a [128 rows][64 bf16] swizzled slab
constexpr int MAX_RING = 4;
constexpr float RESCALE_THRESHOLD = 8.f;  // log2 units
constexpr int SMEM_LIMIT = 232448;
constexpr int SMEM_EXTRA = 1024 + 512;  // start on a 1024-byte boundary; barriers

__device__ int g_error_word = 0;

struct Params {
  const int* block_table;
  int table_width;
  const int *req_indptr, *kv_before, *tile_req, *tile_row;
  __nv_bfloat16* out;  // [tokens][out_stride]: head h at h * v_cols
  long long out_stride;
  int nh, nkv, page_size, window, keep, chunks, v_cols, rows_per_tile;
  int k_ring, v_ring;  // slots
  int stream_q;        // the query pieces come with every K tile
  float scale_log2;
};

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float max3(float a, float b, float c) {
  float r;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(r) : "f"(a), "f"(b), "f"(c));
  return r;
}
__device__ __forceinline__ void fence_proxy_async() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }

// O += P V: A (P) K-major, B (V) MN-major (bit 16).
template <int P> __device__ __forceinline__ uint32_t idesc_pv() { return idesc_bf16_f32(ROWS, P) | (1u << 16); }
// The MN-major operand V: one or two slabs (64 entries of the head each) of [128 keys][64]; 8 keys form a 1024-byte swizzle
// atom (stride byte offset), the slabs are SLAB bytes apart (leading byte offset).
__device__ __forceinline__ uint64_t smem_desc_v(uint32_t saddr) {
  uint64_t desc = 0;
  desc |= (uint64_t)((saddr & 0x3FFFF) >> 4);
  desc |= (uint64_t)(SLAB >> 4) << 16;
  desc |= (uint64_t)(1024 >> 4) << 32;
  desc |= (uint64_t)1 << 46;
  desc |= (uint64_t)2 << 61;
  return desc;
}
// D (+)= A B with A in tensor memory (row i in lane i, two bfloat16 of consecutive k a 32-bit column).
__device__ __forceinline__ void mma_bf16_a_tmem(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b, uint32_t idesc,
                                                bool accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}\n" ::"r"(tmem_d),
      "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"((uint32_t)accumulate)
      : "memory");
}
__device__ __forceinline__ void tmem_st_32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};" ::"r"(taddr),
      "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
      "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]),
      "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]),
      "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// The key tiles of a CTA: ``kept`` tiles from position 0 on, then the tiles from ``first`` on.
struct Walk {
  int kept, first, count, lo, hi, keep;
  __device__ __forceinline__ int tile(int i) const { return i < kept ? i : first + (i - kept); }
  // Whole pages are copied, so a tile may hold rows of keys no row of the CTA sees (pages given back, page 0, keys beyond the
  // last): whatever those pages held before.  Their weights are exactly 0, but 0 x NaN is NaN.
  __device__ __forceinline__ bool dead(int key) const { return key > hi || (key < lo && key >= keep); }
  __device__ __forceinline__ bool edge(int i) const {
    const int k0 = tile(i) * KEYS, k1 = k0 + KEYS - 1;
    return k1 > hi || max(k0, keep) <= min(k1, lo - 1);
  }
};

template <int P>
__global__ void __launch_bounds__(THREADS, 1)
attention_spread_kernel(const __grid_constant__ CUtensorMap map_kv, const __grid_constant__ CUtensorMap map_q, const Params p) {
  constexpr int TILE_BYTES = (P / 64) * SLAB;
  constexpr int SLABS = P / 64;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int k_slot_bytes = TILE_BYTES * (p.stream_q ? 2 : 1);  // with streamed queries: K, then the query piece
  uint8_t* q_tiles = smem;
  uint8_t* k_tiles = q_tiles + (p.stream_q ? 0 : p.chunks * TILE_BYTES);
  uint8_t* v_tiles = k_tiles + p.k_ring * k_slot_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_tiles + p.v_ring * TILE_BYTES);
  uint64_t* k_full = bars;                 // [MAX_RING]
  uint64_t* k_empty = bars + MAX_RING;
  uint64_t* v_full = bars + 2 * MAX_RING;
  uint64_t* v_empty = bars + 3 * MAX_RING;
  uint64_t* s_full = bars + 4 * MAX_RING;  // [2] S of a key tile is in tensor memory
  uint64_t* p_full = s_full + 2;           // [2] (4 arrivals: one a softmax warp) P is written
  uint64_t* pv_done = s_full + 4;          // P V of a key tile is done
  uint64_t* v_clean = s_full + 5;          // [2 V slots] value rows no row sees are cleared (edge tiles)
  uint64_t* q_full = s_full + 7;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(s_full + 8);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kvh = blockIdx.x;
  const int req = p.tile_req[blockIdx.y];
  const int g = p.nh / p.nkv;
  const int tok0 = p.req_indptr[req];
  const int q_len = p.req_indptr[req + 1] - tok0;
  const int before = p.kv_before[req];
  const int* table = p.block_table + (size_t)req * p.table_width;
  const int row_start = p.tile_row[blockIdx.y];
  const int row_end = min(q_len * g, row_start + p.rows_per_tile);
  Walk walk;
  walk.keep = p.keep;
  walk.kept = walk.count = walk.first = walk.lo = 0;
  walk.hi = -1;
  if (row_start < row_end) {
    walk.lo = tl::first_key(before + row_start / g, p.window);
    walk.hi = before + (row_end - 1) / g;
    walk.first = walk.lo / KEYS;
    walk.kept = min((p.keep + KEYS - 1) / KEYS, walk.first);
    walk.count = walk.kept + walk.hi / KEYS + 1 - walk.first;
  }
  const int count = walk.count;

  if (threadIdx.x == 0) {
    for (int i = 0; i < MAX_RING; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&p_full[i], 4);
      mbar_init(&v_clean[i], 1);
    }
    mbar_init(pv_done, 1);
    mbar_init(q_full, 1);
    *abort_flag = 0;
    mbar_fence_init();
    prefetch_tensormap(&map_kv);
    prefetch_tensormap(&map_q);
  }
  if (warp == 4) {
    tmem_alloc<512>(tmem_slot);
    tmem_relinquish();
  }
  tl::pdl_wait();
  tl::pdl_launch_dependents();
  fence_before_sync();
  __syncthreads();
  fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;
  const int pages_per_tile = KEYS / p.page_size;

  if (warp == 5) {
    // ------------------------------------------------------------ K (and Q) loader
    // a query piece: SLABS boxes of [tokens][heads of the group][64 entries]; rows beyond the step's tokens read as zero,
    // rows of the next request's tokens are computed and never stored
    const uint32_t q_bytes = (uint32_t)p.rows_per_tile * 128 * SLABS;
    auto load_q = [&](uint8_t* dst, int c, uint64_t* bar) {  // (lanes below SLABS)
      tma_load_3d(dst + lane * SLAB, &map_q, bar, c * P + lane * 64, kvh * g, tok0 + row_start / g);
    };
    if (!p.stream_q && count > 0) {
      if (lane == 0) mbar_expect_tx(q_full, q_bytes * p.chunks);
      __syncwarp();
      if (lane < SLABS)
        for (int c = 0; c < p.chunks; ++c) load_q(q_tiles + c * TILE_BYTES, c, q_full);
    }
    const int my_page = lane / SLABS, my_slab = lane % SLABS;
    const bool active = my_page < pages_per_tile;
    int item = 0, slot = 0;
    uint32_t phase = 0;
    for (int i = 0; i < count; ++i) {
      const int index = walk.tile(i) * pages_per_tile + my_page;
      const int page = (active && index < p.table_width) ? table[index] : 0;  // beyond the table: page 0
      for (int c = 0; c < p.chunks; ++c, ++item) {
        const int head = p.chunks > 1 ? c : kvh;
        mbar_wait(&k_empty[slot], phase ^ 1, abort_flag, &g_error_word, 1);
        if (lane == 0) mbar_expect_tx(&k_full[slot], TILE_BYTES + (p.stream_q ? q_bytes : 0));
        __syncwarp();
        uint8_t* dst = k_tiles + slot * k_slot_bytes;
        if (active)
          tma_load_2d(dst + my_slab * SLAB + my_page * p.page_size * 128, &map_kv, &k_full[slot], my_slab * 64,
                      (page * 2 * p.nkv + head) * p.page_size);
        if (p.stream_q && lane < SLABS) load_q(dst + TILE_BYTES, c, &k_full[slot]);
        if (++slot == p.k_ring) {
          slot = 0;
          phase ^= 1;
        }
      }
    }
  } else if (warp == 6) {
    // ------------------------------------------------------------------- V loader
    const int my_page = lane / SLABS, my_slab = lane % SLABS;
    const bool active = my_page < pages_per_tile;
    int slot = 0;
    uint32_t phase = 0;
    for (int i = 0; i < count; ++i) {
      const int tile = walk.tile(i);
      const int index = tile * pages_per_tile + my_page;
      const int page = (active && index < p.table_width) ? table[index] : 0;
      uint8_t* dst = v_tiles + slot * TILE_BYTES;
      mbar_wait(&v_empty[slot], phase ^ 1, abort_flag, &g_error_word, 2);
      if (lane == 0) mbar_expect_tx(&v_full[slot], TILE_BYTES);
      __syncwarp();
      if (active)
        tma_load_2d(dst + my_slab * SLAB + my_page * p.page_size * 128, &map_kv, &v_full[slot], my_slab * 64,
                    ((page * 2 + 1) * p.nkv + kvh) * p.page_size);
      if (walk.edge(i)) {
        mbar_wait(&v_full[slot], phase, abort_flag, &g_error_word, 10);  // the tile has landed
        for (int e = lane; e < KEYS * SLABS * 8; e += 32) {  // a key's row: 128 bytes in each slab
          const int k = e / (SLABS * 8);
          if (walk.dead(tile * KEYS + k))
            *reinterpret_cast<uint4*>(dst + ((e >> 3) % SLABS) * SLAB + k * 128 + (e & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
        fence_proxy_async();  // the tensor core reads, and later copies overwrite, what these stores wrote
        __syncwarp();
        if (lane == 0) mbar_arrive(&v_clean[slot]);
      }
      if (++slot == p.v_ring) {
        slot = 0;
        phase ^= 1;
      }
    }
  } else if (warp == 4) {
    // ------------------------------------------------------------------------ MMA
    // The whole warp walks the loop and waits; one elected lane issues.
    const uint32_t idesc_s = idesc_bf16_f32(ROWS, KEYS);
    const uint32_t idesc_o = idesc_pv<P>();
    const uint32_t tmem_o = tmem_base + 256;
    int k_slot = 0, v_slot = 0;
    uint32_t edge_parity = 0;  // a bit a V slot: the parity of its next cleared tile
    uint32_t k_phase = 0, v_phase = 0;
    if (!p.stream_q && count > 0) mbar_wait(q_full, 0, abort_flag, &g_error_word, 4);
    for (int i = 0; i <= count; ++i) {
      if (i < count) {  // S of key tile i; its buffer's P V (tile i - 2) was issued before, and that behind its softmax
        const uint32_t tmem_s = tmem_base + (i & 1) * KEYS;
        for (int c = 0; c < p.chunks; ++c) {
          mbar_wait(&k_full[k_slot], k_phase, abort_flag, &g_error_word, 3);
          fence_after_sync();
          if (elect_one()) {
            const uint8_t* k_tile = k_tiles + k_slot * k_slot_bytes;
            const uint64_t a_desc = smem_desc_sw128(smem_addr(p.stream_q ? k_tile + TILE_BYTES : q_tiles + c * TILE_BYTES));
            const uint64_t b_desc = smem_desc_sw128(smem_addr(k_tile));
#pragma unroll
            for (int k = 0; k < P / 16; ++k) {  // slab k / 4, 32 bytes a slice within its 128-byte rows
              const uint64_t offset = (uint64_t)(((k >> 2) * SLAB + (k & 3) * 32) >> 4);
              mma_bf16(tmem_s, a_desc + offset, b_desc + offset, idesc_s, c > 0 || k > 0);
            }
            mma_commit(&k_empty[k_slot]);
            if (c == p.chunks - 1) mma_commit(&s_full[i & 1]);
          }
          __syncwarp();
          if (++k_slot == p.k_ring) {
            k_slot = 0;
            k_phase ^= 1;
          }
        }
      }
      if (i > 0) {  // O += P V of key tile i - 1
        const int t = i - 1;
        mbar_wait(&v_full[v_slot], v_phase, abort_flag, &g_error_word, 6);
        if (walk.edge(t)) {
          mbar_wait(&v_clean[v_slot], (edge_parity >> v_slot) & 1, abort_flag, &g_error_word, 11);
          edge_parity ^= 1u << v_slot;
        }
        mbar_wait(&p_full[t & 1], (t >> 1) & 1, abort_flag, &g_error_word, 5);
        fence_after_sync();
        if (elect_one()) {
          const uint64_t b_desc = smem_desc_v(smem_addr(v_tiles + v_slot * TILE_BYTES));
          const uint32_t tmem_p = tmem_base + (t & 1) * KEYS;
#pragma unroll
          for (int k = 0; k < KEYS / 16; ++k)  // 16 keys: 8 columns of P, two 8-key atoms of V (2048 bytes)
            mma_bf16_a_tmem(tmem_o, tmem_p + k * 8, b_desc + (uint64_t)(k * (2048 >> 4)), idesc_o, t > 0 || k > 0);
          mma_commit(&v_empty[v_slot]);
          mma_commit(pv_done);
        }
        __syncwarp();
        if (++v_slot == p.v_ring) {
          v_slot = 0;
          v_phase ^= 1;
        }
      }
    }
  } else {
    // -------------------------------------------------------------------- softmax
    const int r = warp * 32 + lane;  // row of the tile = lane of tensor memory
    const int row = row_start + r;
    const bool row_valid = r < p.rows_per_tile && row < row_end;
    const int pos = row_valid ? before + row / g : -1;
    const int lo = row_valid ? tl::first_key(pos, p.window) : 0;
    const int keep_end = min(p.keep, pos + 1);
    const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
    const uint32_t tmem_o = tmem_base + 256 + lane_base;
    float m_ref = -INFINITY, l_sum = 0.f;  // m_ref in log2 units (already scaled)
    for (int t = 0; t < count; ++t) {
      const uint32_t tmem_s = tmem_base + (t & 1) * KEYS + lane_base;
      const int key0 = walk.tile(t) * KEYS;
      mbar_wait(&s_full[t & 1], (t >> 1) & 1, abort_flag, &g_error_word, 7);
      fence_after_sync();
      uint32_t v[KEYS];
#pragma unroll
      for (int c = 0; c < KEYS; c += 32) tmem_ld_32(tmem_s + c, reinterpret_cast<uint32_t(&)[32]>(v[c]));
      tmem_ld_wait();
      // rows beyond the tile's last (never stored) take whatever comes
      const bool visible = !row_valid || (key0 + KEYS - 1 <= pos && (key0 >= lo || key0 + KEYS <= keep_end));
      if (!__all_sync(0xffffffffu, visible)) {
        const int first_rel = lo - key0, keep_rel = keep_end - key0;
        const unsigned span = row_valid ? (unsigned)(pos - lo) : 0x7fffffffu;
#pragma unroll
        for (int i = 0; i < KEYS; ++i) {
          // key0 + i outside [lo, pos] (one unsigned comparison) and not one of the kept ones
          if ((unsigned)(i - first_rel) > span && i >= keep_rel) v[i] = __float_as_uint(-INFINITY);
        }
      }
      float m_a = -INFINITY, m_b = -INFINITY, m_c = -INFINITY, m_d = -INFINITY;
#pragma unroll
      for (int i = 0; i < KEYS; i += 8) {
        m_a = max3(m_a, __uint_as_float(v[i]), __uint_as_float(v[i + 1]));
        m_b = max3(m_b, __uint_as_float(v[i + 2]), __uint_as_float(v[i + 3]));
        m_c = max3(m_c, __uint_as_float(v[i + 4]), __uint_as_float(v[i + 5]));
        m_d = max3(m_d, __uint_as_float(v[i + 6]), __uint_as_float(v[i + 7]));
      }
      const float m_tile = fmaxf(fmaxf(m_a, m_b), fmaxf(m_c, m_d)) * p.scale_log2;  // the factor is positive
      float factor = 1.f;
      bool rescale = false;
      if (m_tile > m_ref + RESCALE_THRESHOLD || (m_ref == -INFINITY && m_tile > -INFINITY)) {
        factor = m_ref == -INFINITY ? 0.f : fast_exp2(m_ref - m_tile);
        rescale = m_ref != -INFINITY;
        m_ref = m_tile;
      }
      l_sum *= factor;
      if (__any_sync(0xffffffffu, rescale)) {  // (never in the first tile)
        // P V of the tile before may still run: the next one cannot start before this tile's P is handed over
        mbar_wait(pv_done, (t - 1) & 1, abort_flag, &g_error_word, 8);
        fence_after_sync();
#pragma unroll 1
        for (int c = 0; c < P; c += 32) {
          uint32_t o[32];
          tmem_ld_32(tmem_o + c, o);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * factor);
          tmem_st_32(tmem_o + c, o);
        }
      }
      // P = exp2(S * scale - m_ref) as bfloat16 pairs over the first half of S's columns; row sum
      const float neg_m = m_ref == -INFINITY ? 0.f : -m_ref;
      float sum_a = 0.f, sum_b = 0.f;
#pragma unroll
      for (int c = 0; c < KEYS; c += 64) {
        uint32_t packed[32];
#pragma unroll
        for (int i = 0; i < 64; i += 2) {
          const float a = fast_exp2(fmaf(__uint_as_float(v[c + i]), p.scale_log2, neg_m));
          const float b = fast_exp2(fmaf(__uint_as_float(v[c + i + 1]), p.scale_log2, neg_m));
          sum_a += a;
          sum_b += b;
          __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
          packed[i >> 1] = *reinterpret_cast<uint32_t*>(&h);
        }
        tmem_st_32(tmem_s + (c >> 1), packed);
      }
      l_sum += sum_a + sum_b;
      tmem_st_wait();
      fence_before_sync();  // our tcgen05.ld/st of S, P and O are done
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[t & 1]);
    }
    if (count > 0) {
      // the last two, in turn: a parity alone does not tell the last P V from the one two before it
      if (count > 1) mbar_wait(pv_done, (count - 2) & 1, abort_flag, &g_error_word, 8);
      mbar_wait(pv_done, (count - 1) & 1, abort_flag, &g_error_word, 9);
      fence_after_sync();
      const float inv = l_sum > 0.f ? 1.f / l_sum : 0.f;
      __nv_bfloat16* dst = p.out;
      if (row_valid) dst = p.out + (size_t)(tok0 + row / g) * p.out_stride + (size_t)(kvh * g + row % g) * p.v_cols;
      const bool wide = p.v_cols % 8 == 0 && p.out_stride % 8 == 0;
#pragma unroll 1
      for (int c = 0; c < P; c += 32) {
        uint32_t o[32];
        tmem_ld_32(tmem_o + c, o);
        tmem_ld_wait();
        if (row_valid) {
          uint32_t packed[16];
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            __nv_bfloat162 h = __floats2bfloat162_rn(__uint_as_float(o[i]) * inv, __uint_as_float(o[i + 1]) * inv);
            packed[i >> 1] = *reinterpret_cast<uint32_t*>(&h);
          }
          if (wide) {
#pragma unroll
            for (int q4 = 0; q4 < 4; ++q4)
              if (c + 8 * q4 < p.v_cols)
                *reinterpret_cast<uint4*>(dst + c + 8 * q4) =
                    make_uint4(packed[4 * q4], packed[4 * q4 + 1], packed[4 * q4 + 2], packed[4 * q4 + 3]);
          } else {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (c + i < p.v_cols) dst[c + i] = __float2bfloat16_rn(__uint_as_float(o[i]) * inv);
          }
        }
      }
    }
  }
  __syncwarp();
  fence_before_sync();
  __syncthreads();
  if (warp == 4) {
    fence_after_sync();
    tmem_dealloc<512>(tmem_base);
  }
}

// ------------------------------------------------------------------ host side
struct MapKey {
  const void* base;
  uint64_t a, b, c;
  uint32_t box_a, box_b;
  bool operator==(const MapKey& o) const {
    return base == o.base && a == o.a && b == o.b && c == o.c && box_a == o.box_a && box_b == o.box_b;
  }
};
struct MapKeyHash {
  size_t operator()(const MapKey& k) const {
    size_t h = reinterpret_cast<size_t>(k.base);
    for (uint64_t x : {k.a, k.b, k.c, (uint64_t)k.box_a, (uint64_t)k.box_b}) h = h * 1000003u ^ x;
    return h;
  }
};
template <typename Make> bool cached_map(CUtensorMap* out, const MapKey& key, Make make) {
  static std::unordered_map<MapKey, CUtensorMap, MapKeyHash> cache;
  static std::mutex lock;
  std::lock_guard<std::mutex> guard(lock);
  auto it = cache.find(key);
  if (it == cache.end()) {
    CUtensorMap map;
    if (!make(&map)) return false;
    if (cache.size() > 1024) cache.clear();
    it = cache.emplace(key, map).first;
  }
  *out = it->second;
  return true;
}

// Queries [tokens][nh][width] bf16 (tokens ``stride`` elements apart): boxes of 64 entries x group heads x box_tokens tokens.
bool make_query_map(CUtensorMap* map, const void* base, uint64_t width, uint64_t nh, uint64_t tokens, uint64_t stride,
                    uint32_t group, uint32_t box_tokens) {
  tc_host::EncodeTiledFn fn = tc_host::encode_fn();
  if (!fn || (reinterpret_cast<uintptr_t>(base) & 15) || (width * 2) % 16 || (stride * 2) % 16) return false;
  cuuint64_t dims[3] = {width, nh, tokens};
  cuuint64_t strides[2] = {width * 2, stride * 2};
  cuuint32_t box[3] = {64, group, box_tokens};
  cuuint32_t elem[3] = {1, 1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, elem,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int P>
int launch(const CUtensorMap& map_kv, const CUtensorMap& map_q, Params p, int tiles, cudaStream_t stream) {
  constexpr int TILE_BYTES = (P / 64) * SLAB;
  const int room = (SMEM_LIMIT - SMEM_EXTRA) / TILE_BYTES;  // operand tiles: 7 for P = 128, 14 for P = 64
  if (p.chunks + 3 <= room) {
    p.stream_q = 0;
    const int left = room - p.chunks;  // at least two K slots and one V slot
    p.v_ring = left >= 4 ? 2 : 1;
    p.k_ring = left - p.v_ring < MAX_RING ? left - p.v_ring : MAX_RING;
  } else {
    p.stream_q = 1;
    p.v_ring = 2;
    p.k_ring = 2;
  }
  const int smem = ((p.stream_q ? 0 : p.chunks) + p.k_ring * (p.stream_q ? 2 : 1) + p.v_ring) * TILE_BYTES + SMEM_EXTRA;
  if (smem > SMEM_LIMIT) return TL_ERR_UNSUPPORTED;
  static bool configured = false;
  if (!configured) {
    cudaError_t err = cudaFuncSetAttribute(attention_spread_kernel<P>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_LIMIT);
    if (err != cudaSuccess) return (int)err;
    configured = true;
  }
  tl::launch_kernel(attention_spread_kernel<P>, dim3(p.nkv, tiles), THREADS, smem, stream, map_kv, map_q, p);
  return TL_LAUNCH_CHECK();
}

}  // namespace

extern "C" {

int tl_attention_spread_error() {
  int value = 0, zero = 0;
  if (cudaMemcpyFromSymbol(&value, g_error_word, sizeof(int)) != cudaSuccess) return -1;
  if (value) cudaMemcpyToSymbol(g_error_word, &zero, sizeof(int));
  return value;
}

// Packed rows a CTA takes for a group of ``group`` query heads: whole tokens.
int tl_attention_spread_rows(int group) { return group > 0 && group <= ROWS ? (ROWS / group) * group : 0; }

// q [tokens][nh][chunks p] bf16 rows (q_stride elements apart); chunks 1 or nkv.  pages: one cache layer
// [num_pages][2][nkv][page_size][p] bf16, p 64 or 128.  tile_req / tile_row: request and first packed row (a multiple of
// tl_attention_spread_rows(nh / nkv)) of each CTA.  out [tokens][out_stride]: v_cols entries a head.
int tl_attention_spread(const void* q, long long q_stride, const void* pages, long long num_pages, const int* block_table,
                        int table_width, const int* req_indptr, const int* kv_before, const int* tile_req, const int* tile_row,
                        int tiles, void* out, long long out_stride, int tokens, int nh, int nkv, int p_size, int page_size,
                        int window, int keep, int chunks, int v_cols, float scale, cudaStream_t stream) {
  if (tiles <= 0) return 0;
  if ((p_size != 64 && p_size != 128) || nkv <= 0 || nh % nkv || nh / nkv > ROWS || page_size < 8 || page_size > KEYS ||
      KEYS % page_size || q_stride % 8 || tiles > 65535 || !tile_req || !tile_row || keep < 0 || v_cols <= 0 || v_cols > p_size ||
      (chunks != 1 && chunks != nkv) || !(scale > 0.f))
    return TL_ERR_UNSUPPORTED;
  const int group = nh / nkv;
  CUtensorMap map_kv, map_q;
  const uint64_t kv_rows = (uint64_t)num_pages * 2 * nkv * page_size;
  if (!cached_map(&map_kv, MapKey{pages, kv_rows, (uint64_t)p_size, 0, (uint32_t)page_size, 0},
                  [&](CUtensorMap* m) { return tc_host::make_map_bf16(m, pages, kv_rows, p_size, p_size, page_size); }))
    return TL_ERR_UNSUPPORTED;
  const uint64_t width = (uint64_t)chunks * p_size;
  const uint32_t box_tokens = ROWS / group;
  const MapKey q_key{q, width | ((uint64_t)nh << 32), (uint64_t)tokens, (uint64_t)q_stride, (uint32_t)group, box_tokens};
  if (!cached_map(&map_q, q_key,
                  [&](CUtensorMap* m) { return make_query_map(m, q, width, nh, tokens, q_stride, group, box_tokens); }))
    return TL_ERR_UNSUPPORTED;
  Params p;
  memset(&p, 0, sizeof(p));
  p.block_table = block_table;
  p.table_width = table_width;
  p.req_indptr = req_indptr;
  p.kv_before = kv_before;
  p.tile_req = tile_req;
  p.tile_row = tile_row;
  p.out = (__nv_bfloat16*)out;
  p.out_stride = out_stride;
  p.nh = nh;
  p.nkv = nkv;
  p.page_size = page_size;
  p.window = window;
  p.keep = window > 0 ? keep : 0;
  p.chunks = chunks;
  p.v_cols = v_cols;
  p.rows_per_tile = tl_attention_spread_rows(group);
  p.scale_log2 = scale * 1.4426950408889634f;
  return p_size == 128 ? launch<128>(map_kv, map_q, p, tiles, stream) : launch<64>(map_kv, map_q, p, tiles, stream);
}

}  // extern "C"
