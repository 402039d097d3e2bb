// Latent attention of portions of prompts on the 5th-generation tensor cores (bfloat16), with every head's keys and values
// multiplied out of the cached latents first: a portion's query then meets dim + rot entries of a key instead of the latent's
// whole width, a third of the work for a latent of 512.
//
// latent_gather_kernel copies the cached vectors [c | rotated key part] of the portions' requests out of their pages, one
// row a position, zeros behind a request's last position; an ordinary product turns the rows' latents into
// kv [rows, heads * dim (keys) | heads * vdim (values)]; latent_prefill_kernel attends.
//
// latent_prefill_kernel is attention_tcgen05.cu's kernel with other operands (see there for the softmax by one thread a query
// row, the reference that follows the maximum, P in tensor memory and the order of the products).  A work item is a run of
// up to 256 tokens of one request for ONE head: two tiles of 128 query rows that share the keys and values the CTA loads.
//     S = Q_u K_u^T + Q_r K_r^T    K_u: the head's columns of kv, in chunks of 64 entries; K_r: the rotated part, the same
//                                  columns of the gathered rows for every head
//     O += P V                     V: the head's value columns of kv
// All operands come through TMA in boxes of 64 entries x 64 rows (queries: x 128), 128-byte swizzle.  Where a head's size is
// no multiple of 64 a chunk of keys runs into the columns behind it; the queries' chunk reads zeros there, so these add
// nothing, and value columns behind the head's are not stored.  Rows behind a request's last position are zeros or another
// request's rows: finite, and masked.
//
// A learned sink joins a row's sum at the end, and the head's gate multiplies the row before the one rounding.  gridDim.z > 1
// cuts the blocks of an item into ranges that latent_prefill_combine_kernel adds up in their order.
#include "attention_tcgen05.cuh"

#include <unordered_map>

namespace lb {

struct LatentPrefillParams {
  bf16* out;                                // [T, heads, vdim]
  const int* positions;
  const int4* tiles;                        // {first token, tokens, unused, first row of the request in kv}
  const float* sinks;                       // optional [heads]
  const float* gate; long long ldg;         // optional [T, heads], row stride ldg
  int heads, dim, rot, vdim, kv_rank, dim_chunks, chunks;      // chunks: of a key, the rotated one included
  float scale_log2;
  float* part_o; float* part_ml;            // [(item * heads + head) * ranges + range][TA_PART_ROWS][vdim | 2]
};

enum : int { LP_ERR_Q = 601, LP_ERR_KV_FULL = 602, LP_ERR_KV_EMPTY = 603, LP_ERR_S_FULL = 604, LP_ERR_P_FULL = 606, LP_ERR_O_FULL = 608 };

constexpr int LP_MAX_CHUNKS = 3;                                  // chunks of 64 entries of a query or key
constexpr int LP_STAGES = 3;
constexpr int LP_BOX = TA_KEYS * 128;                             // 64 rows of 64 entries: 8 KB
constexpr int LP_Q_TILE = LP_MAX_CHUNKS * TA_HALF_BYTES;          // a tile of queries: 48 KB
constexpr int LP_K_STAGE = LP_MAX_CHUNKS * LP_BOX, LP_V_STAGE = 2 * LP_BOX;
constexpr int LP_K_OFF = 2 * LP_Q_TILE;
constexpr int LP_V_OFF = LP_K_OFF + LP_STAGES * LP_K_STAGE;
constexpr int LP_BAR_OFF = LP_V_OFF + LP_STAGES * LP_V_STAGE;
constexpr int LP_NUM_BARS = 1 + 4 * LP_STAGES + 2 * 6;
constexpr int LP_SMEM_BYTES = LP_BAR_OFF + LP_NUM_BARS * 8 + 16;
constexpr int LP_THREADS = 384;

__device__ __forceinline__ void lp_tma_2d(uint32_t dst, const CUtensorMap* map, int x, int y, uint32_t bar) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
               ::"r"(dst), "l"(map), "r"(x), "r"(y), "r"(bar) : "memory");
}

// VC: chunks of 64 entries of a value head.
template <int VC>
__global__ void __launch_bounds__(LP_THREADS, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap map_qu, const __grid_constant__ CUtensorMap map_qr,
                      const __grid_constant__ CUtensorMap map_kv, const __grid_constant__ CUtensorMap map_lat, LatentPrefillParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  const uint32_t sbase = ta_smem_u32(smem);
  const uint32_t bars = sbase + LP_BAR_OFF;
  const uint32_t q_full = bars;
  auto k_full = [&](int s) { return bars + 8u * (1 + s); };
  auto k_empty = [&](int s) { return bars + 8u * (1 + LP_STAGES + s); };
  auto v_full = [&](int s) { return bars + 8u * (1 + 2 * LP_STAGES + s); };
  auto v_empty = [&](int s) { return bars + 8u * (1 + 3 * LP_STAGES + s); };
  // per tile t and S buffer b: S complete, P written, P V complete
  auto s_full = [&](int t, int b) { return bars + 8u * (1 + 4 * LP_STAGES + t * 6 + b); };
  auto p_full = [&](int t, int b) { return bars + 8u * (1 + 4 * LP_STAGES + t * 6 + 2 + b); };
  auto pv_done = [&](int t, int b) { return bars + 8u * (1 + 4 * LP_STAGES + t * 6 + 4 + b); };
  uint32_t* tmem_slot = (uint32_t*)(smem + LP_BAR_OFF + LP_NUM_BARS * 8);
  volatile int* abort_flag = (volatile int*)(tmem_slot + 1);

  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int4 tile = p.tiles[blockIdx.y];        // heads run fastest: the items come heaviest first over the whole grid
  const int t0 = tile.x, ntok = tile.y, row0 = tile.w;
  const int head = blockIdx.x;
  const bool two = ntok > TA_ROWS;
  const int ntiles = two ? 2 : 1;

  if (threadIdx.x == 0) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(&map_qu) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&map_kv) : "memory");
    ta_mbar_init(q_full, 1);
    for (int i = 0; i < LP_STAGES; ++i) {
      ta_mbar_init(k_full(i), 1); ta_mbar_init(k_empty(i), ntiles);       // a stage goes back when every tile's product has read it
      ta_mbar_init(v_full(i), 1); ta_mbar_init(v_empty(i), ntiles);
    }
    for (int t = 0; t < 2; ++t)
      for (int b = 0; b < 2; ++b) { ta_mbar_init(s_full(t, b), 1); ta_mbar_init(p_full(t, b), 4); ta_mbar_init(pv_done(t, b), 1); }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(ta_smem_u32(tmem_slot)), "r"(512) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = *tmem_slot;            // columns: tile t's S buffers at t * 128 and t * 128 + 64 (P over their first 32), O at 256 + t * 128

  const int pos0 = p.positions[t0];             // written before the step began
  const int kend_all = pos0 + ntok;             // exclusive
  const int nblocks_all = (kend_all + TA_KEYS - 1) / TA_KEYS;
  const int nsplit = gridDim.z, isplit = blockIdx.z;
  const int blk0 = (int)((long long)nblocks_all * isplit / nsplit), blk1 = (int)((long long)nblocks_all * (isplit + 1) / nsplit);
  const int kbeg = blk0 * TA_KEYS;
  const int nblocks = blk1 - blk0;              // a range may be empty when the item sees few keys
  pdl_wait();                                   // the queries, keys and values below are what earlier kernels wrote

  if (nblocks <= 0) {
    if (warp >= 2 && warp < 10) {               // its rows weigh nothing in the combination
      const int r = ((warp - 2) >> 2) * TA_ROWS + (warp & 3) * 32 + lane;
      if (r < ntok) {
        const size_t prow = (((size_t)blockIdx.y * p.heads + head) * nsplit + isplit) * TA_PART_ROWS + r;
        p.part_ml[prow * 2] = -INFINITY;
        p.part_ml[prow * 2 + 1] = 0.f;
      }
    }
  } else if (warp == 0 || warp == 10) {
    // ---- producers, a thread each: warp 0 the queries and the keys, warp 10 the values -----------------------------------
    if (lane == 0) {
      const bool is_v = warp == 10;
      if (!is_v) {
        ta_mbar_expect_tx(q_full, (uint32_t)(ntiles * p.chunks) * TA_HALF_BYTES);
        for (int t = 0; t < ntiles; ++t)
          for (int c = 0; c < p.chunks; ++c) {
            const uint32_t dst = sbase + t * LP_Q_TILE + c * TA_HALF_BYTES;
            if (c < p.dim_chunks) ta_tma_3d(dst, &map_qu, c * 64, head, t0 + t * TA_ROWS, q_full);
            else ta_tma_3d(dst, &map_qr, 0, head, t0 + t * TA_ROWS, q_full);
          }
      }
      int i = 0;
      for (; i < nblocks; ++i) {
        const int s = i % LP_STAGES;
        if (!ta_mbar_wait_idle(is_v ? v_empty(s) : k_empty(s), (uint32_t)((i / LP_STAGES) & 1) ^ 1u, abort_flag, LP_ERR_KV_EMPTY)) break;
        const int y = row0 + kbeg + i * TA_KEYS;
        if (is_v) {
          ta_mbar_expect_tx(v_full(s), VC * LP_BOX);
          for (int c = 0; c < VC; ++c)
            lp_tma_2d(sbase + LP_V_OFF + s * LP_V_STAGE + c * LP_BOX, &map_kv, p.heads * p.dim + head * p.vdim + c * 64, y, v_full(s));
        } else {
          ta_mbar_expect_tx(k_full(s), (uint32_t)p.chunks * LP_BOX);
          for (int c = 0; c < p.chunks; ++c) {
            const uint32_t dst = sbase + LP_K_OFF + s * LP_K_STAGE + c * LP_BOX;
            if (c < p.dim_chunks) lp_tma_2d(dst, &map_kv, head * p.dim + c * 64, y, k_full(s));
            else lp_tma_2d(dst, &map_lat, p.kv_rank, y, k_full(s));
          }
        }
      }
      // nobody leaves while a copy of its own is in flight
      for (int j = max(0, i - LP_STAGES); j < i; ++j)
        ta_mbar_wait_idle(is_v ? v_full(j % LP_STAGES) : k_full(j % LP_STAGES), (uint32_t)((j / LP_STAGES) & 1), abort_flag, LP_ERR_KV_FULL);
      if (!is_v) ta_mbar_wait_idle(q_full, 0, abort_flag, LP_ERR_Q);
    }
  } else if (warp == 1 || warp == 11) {
    // ---- tensor-core issue, one thread per tile --------------------------------------------------------------
    const int t = warp == 1 ? 0 : 1;
    if (lane == 0 && t < ntiles) {
      constexpr uint32_t idesc_qk = ta_idesc(0, TA_KEYS), idesc_pv = ta_idesc(1, VC * 64);
      const uint32_t s_col = tmem + (uint32_t)t * 128u, o_col = tmem + 256u + (uint32_t)t * 128u;
      const uint32_t qa = sbase + t * LP_Q_TILE;
      bool ok = ta_mbar_wait(q_full, 0, abort_flag, LP_ERR_Q);
      // S(j) = Q K(j)^T into S buffer j & 1; the keys' stage goes back when every tile's product is done
      auto issue_qk = [&](int j) -> bool {
        const int s = j % LP_STAGES;
        if (!ta_mbar_wait(k_full(s), (uint32_t)((j / LP_STAGES) & 1), abort_flag, LP_ERR_KV_FULL)) return false;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint32_t ka = sbase + LP_K_OFF + s * LP_K_STAGE;
        for (int c = 0; c < p.chunks; ++c)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            ta_umma(s_col + (uint32_t)(j & 1) * 64u, ta_desc_kmajor(qa + (uint32_t)c * TA_HALF_BYTES + (uint32_t)k * 32u),
                    ta_desc_kmajor(ka + (uint32_t)c * LP_BOX + (uint32_t)k * 32u), idesc_qk, (c | k) != 0);
        ta_commit(s_full(t, j & 1));
        ta_commit(k_empty(s));
        return true;
      };
      for (int j = 0; j < 2 && j < nblocks && ok; ++j) ok = issue_qk(j);
      for (int i = 0; i < nblocks && ok; ++i) {
        const int s = i % LP_STAGES, b = i & 1;
        // O += P(i) V(i)
        ok = ta_mbar_wait(p_full(t, b), (uint32_t)((i >> 1) & 1), abort_flag, LP_ERR_P_FULL);
        if (!ok) break;
        ok = ta_mbar_wait(v_full(s), (uint32_t)((i / LP_STAGES) & 1), abort_flag, LP_ERR_KV_FULL);
        if (!ok) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint32_t va = sbase + LP_V_OFF + s * LP_V_STAGE;
#pragma unroll
        for (int k = 0; k < TA_KEYS / 16; ++k)            // 16 keys a step: 8 columns of P, 16 rows of V
          ta_umma_ts(o_col, s_col + (uint32_t)b * 64u + (uint32_t)k * 8u, ta_desc_mnmajor(va + (uint32_t)k * 16u * 128u, LP_BOX),
                     idesc_pv, (i | k) != 0);
        ta_commit(pv_done(t, b));
        ta_commit(v_empty(s));
        // S(i+2) goes where P(i) lies: issued behind P V(i), which the tensor cores finish first
        if (i + 2 < nblocks) ok = issue_qk(i + 2);
      }
    }
  } else if (warp < 6 || (two && warp < 10)) {
    // ---- softmax: warps 2..5 tile A, warps 6..9 tile B; warp w reads lanes (w % 4) * 32 .. + 31 of tensor memory;
    // thread = query row -------------------------------------------------------------------------------------
    const int t = (warp - 2) >> 2;
    const int quarter = warp & 3;
    const int row = t * TA_ROWS + quarter * 32 + lane;       // token of the item
    const uint32_t tlane = (uint32_t)(quarter * 32) << 16;
    const uint32_t s_addr = tmem + tlane + (uint32_t)t * 128u, o_addr = tmem + tlane + 256u + (uint32_t)t * 128u;
    const bool row_valid = row < ntok;
    const int row_pos = row_valid ? pos0 + row : -1;
    const int tile_pos0 = pos0 + t * TA_ROWS;                // the smallest position among the tile's rows
    float m_ref = -INFINITY, l_run = 0.f;
    bool ok = true;

    for (int i = 0; i < nblocks; ++i) {
      const int b = i & 1;
      const int kb = kbeg + i * TA_KEYS;
      ok = ta_mbar_wait(s_full(t, b), (uint32_t)((i >> 1) & 1), abort_flag, LP_ERR_S_FULL);
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      float x[TA_KEYS];
      {
        uint32_t v[64];
        ta_tmem_ld64(s_addr + (uint32_t)b * 64u, v);
#pragma unroll
        for (int j = 0; j < 64; ++j) x[j] = __uint_as_float(v[j]);
      }
      if (kb + TA_KEYS - 1 > tile_pos0) {
#pragma unroll
        for (int j = 0; j < TA_KEYS; ++j)
          if (kb + j > row_pos) x[j] = -INFINITY;
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};      // four chains of three-input maxima
#pragma unroll
      for (int j = 0; j < TA_KEYS; j += 8) {
#pragma unroll
        for (int u = 0; u < 4; ++u) mx4[u] = ta_max3(mx4[u], x[j + 2 * u], x[j + 2 * u + 1]);
      }
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      const float m_loc = mx * p.scale_log2;
      const bool grow = m_loc > m_ref + TA_RESCALE_STEP;      // also true for the first finite maximum (m_ref = -inf)
      if (__any_sync(0xffffffffu, grow)) {
        float f = 1.f;
        if (grow) {
          if (m_ref != -INFINITY) f = exp2f(m_ref - m_loc);
          m_ref = m_loc;
          l_run *= f;
        }
        if (i > 0) {
          ok = ta_mbar_wait(pv_done(t, b ^ 1), (uint32_t)(((i - 1) >> 1) & 1), abort_flag, LP_ERR_O_FULL);
          if (!ok) break;
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll 1
          for (int c = 0; c < VC * 64; c += 32) {
            uint32_t v[32];
            ta_tmem_ld32(o_addr + (uint32_t)c, v);
#pragma unroll
            for (int j = 0; j < 32; ++j) v[j] = __float_as_uint(__uint_as_float(v[j]) * f);
            ta_tmem_st32(o_addr + (uint32_t)c, v);
          }
          ta_tmem_wait_st();
        }
      }
      const float m_use = m_ref == -INFINITY ? 0.f : m_ref;
      const uint64_t scale2 = ta_pack2(p.scale_log2, p.scale_log2), negm2 = ta_pack2(-m_use, -m_use);
      uint64_t sum2 = ta_pack2(0.f, 0.f);
      uint32_t w[32];
#pragma unroll
      for (int j = 0; j < 32; ++j) {
        float y0 = x[2 * j], y1 = x[2 * j + 1];
        ta_unpack2(ta_fma2(ta_pack2(y0, y1), scale2, negm2), y0, y1);
        const float p0 = exp2_approx(y0), p1 = exp2_approx(y1);          // 2^-inf = 0 for masked keys
        sum2 = ta_add2(sum2, ta_pack2(p0, p1));
        __nv_bfloat162 b2 = __floats2bfloat162_rn(p0, p1);
        w[j] = *reinterpret_cast<uint32_t*>(&b2);
      }
      ta_tmem_st32(s_addr + (uint32_t)b * 64u, w);
      ta_tmem_wait_st();
      {
        float s0, s1;
        ta_unpack2(sum2, s0, s1);
        l_run += s0 + s1;
      }
      // hand P to the tensor cores
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0) ta_mbar_arrive(p_full(t, b));
    }
    if (ok) ok = ta_mbar_wait(pv_done(t, (nblocks - 1) & 1), (uint32_t)(((nblocks - 1) >> 1) & 1), abort_flag, LP_ERR_O_FULL);
    if (ok) {
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const int token = t0 + row;
      const size_t prow = (((size_t)blockIdx.y * p.heads + head) * nsplit + isplit) * TA_PART_ROWS + row;
      float f = 1.f;
      if (nsplit > 1) {
        if (row_valid) { p.part_ml[prow * 2] = m_ref; p.part_ml[prow * 2 + 1] = l_run; }
      } else {
        float den = l_run;
        if (p.sinks) {
          const float sink = p.sinks[head] * 1.4426950408889634f, top = fmaxf(m_ref, sink);
          f = m_ref == -INFINITY ? 0.f : exp2f(m_ref - top);
          den = l_run * f + exp2f(sink - top);
        }
        f = den > 0.f ? f / den : 0.f;
        if (p.gate && row_valid) f *= 1.f / (1.f + expf(-p.gate[(size_t)token * p.ldg + head]));
      }
      bf16* dst = p.out + ((size_t)token * p.heads + head) * p.vdim;
#pragma unroll 1
      for (int c = 0; c < VC * 64; c += 32) {
        uint32_t v[32];
        __syncwarp();
        ta_tmem_ld32(o_addr + (uint32_t)c, v);              // warp-wide: rows without a token take part and write nothing
#pragma unroll
        for (int q8 = 0; q8 < 4; ++q8) {                    // a value head's size is a multiple of 8
          if (!row_valid || c + 8 * q8 >= p.vdim) {
          } else if (nsplit > 1) {
            uint4* pdst = reinterpret_cast<uint4*>(p.part_o + prow * p.vdim + c + 8 * q8);
            pdst[0] = make_uint4(v[8 * q8], v[8 * q8 + 1], v[8 * q8 + 2], v[8 * q8 + 3]);
            pdst[1] = make_uint4(v[8 * q8 + 4], v[8 * q8 + 5], v[8 * q8 + 6], v[8 * q8 + 7]);
          } else {
            uint32_t w[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              __nv_bfloat162 b2 = __floats2bfloat162_rn(__uint_as_float(v[8 * q8 + 2 * j]) * f, __uint_as_float(v[8 * q8 + 2 * j + 1]) * f);
              w[j] = *reinterpret_cast<uint32_t*>(&b2);
            }
            *reinterpret_cast<uint4*>(dst + c + 8 * q8) = make_uint4(w[0], w[1], w[2], w[3]);
          }
        }
      }
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 1) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512) : "memory");
  }
}

// The rows of items whose keys were cut into ranges: out = gate * sum_z 2^(m_z - M) o_z / (sum_z 2^(m_z - M) l_z + 2^(sink - M)).
// One warp a row, a lane adds up four entries.  A range without keys for a row is left out: its o_z may never have been written.
constexpr int LP_MAX_SPLITS = 8;
__global__ void __launch_bounds__(256) latent_prefill_combine_kernel(LatentPrefillParams p, int nsplit) {
  pdl_trigger();
  pdl_wait();
  const int4 tile = p.tiles[blockIdx.x];
  const int head = blockIdx.y, lane = threadIdx.x;
  const size_t base = ((size_t)blockIdx.x * p.heads + head) * nsplit;
  for (int r = blockIdx.z * blockDim.y + threadIdx.y; r < tile.y; r += blockDim.y * gridDim.z) {
    const float sink = p.sinks ? p.sinks[head] * 1.4426950408889634f : -INFINITY;
    float w[LP_MAX_SPLITS], M = sink;
#pragma unroll
    for (int z = 0; z < LP_MAX_SPLITS; ++z) {
      w[z] = z < nsplit ? __ldcg(p.part_ml + ((base + z) * TA_PART_ROWS + r) * 2) : -INFINITY;
      M = fmaxf(M, w[z]);
    }
    float L = sink == -INFINITY ? 0.f : exp2f(sink - M);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int z = 0; z < LP_MAX_SPLITS; ++z) {
      if (z < nsplit && w[z] != -INFINITY) {
        const float wz = exp2f(w[z] - M);
        L += __ldcg(p.part_ml + ((base + z) * TA_PART_ROWS + r) * 2 + 1) * wz;
        if (lane * 4 < p.vdim) {
          const float4 a = __ldcg(reinterpret_cast<const float4*>(p.part_o + ((base + z) * TA_PART_ROWS + r) * p.vdim) + lane);
          acc.x += a.x * wz; acc.y += a.y * wz; acc.z += a.z * wz; acc.w += a.w * wz;
        }
      }
    }
    const int token = tile.x + r;
    float f = L > 0.f ? 1.f / L : 0.f;
    if (p.gate) f *= 1.f / (1.f + expf(-p.gate[(size_t)token * p.ldg + head]));
    if (lane * 4 >= p.vdim) continue;
    __nv_bfloat162 lo = __floats2bfloat162_rn(acc.x * f, acc.y * f), hi = __floats2bfloat162_rn(acc.z * f, acc.w * f);
    *reinterpret_cast<uint2*>(p.out + ((size_t)token * p.heads + head) * p.vdim + lane * 4) =
        make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
  }
}

// Row first + j of out = the cached vector of position j of request seq, for entries {seq, first row, rows, unused}; zeros where the
// request has no such position.  A warp a row.
__global__ void __launch_bounds__(256) latent_gather_kernel(uint4* __restrict__ out, const uint4* __restrict__ pool, const int4* __restrict__ entries,
                                                            int num_entries, int total_rows, const int* __restrict__ context_lens,
                                                            const int* __restrict__ block_table, int max_pages, int page_size, int words) {
  pdl_trigger();
  const int lane = threadIdx.x & 31, row = blockIdx.x * 8 + (threadIdx.x >> 5);
  int e = 0;
  int4 en = make_int4(0, 0, 0, 0);
  if (row < total_rows)
    for (; e < num_entries; ++e) {
      en = entries[e];
      if (row < en.y + en.z) break;
    }
  const int j = row - en.y;
  int page = -1;
  if (row < total_rows && e < num_entries && j < context_lens[en.x]) page = block_table[(size_t)en.x * max_pages + j / page_size];
  pdl_wait();
  if (row >= total_rows) return;
  const uint4* src = page >= 0 ? pool + ((size_t)page * page_size + j % page_size) * words : nullptr;
  for (int i = lane; i < words; i += 32) out[(size_t)row * words + i] = src ? src[i] : make_uint4(0u, 0u, 0u, 0u);
}

// ---- host side ------------------------------------------------------------------------------------------------
struct LpMapKey {
  const void* base; long long a, b, c; int kind;
  bool operator==(const LpMapKey& o) const { return base == o.base && a == o.a && b == o.b && c == o.c && kind == o.kind; }
};
struct LpMapKeyHash {
  size_t operator()(const LpMapKey& k) const {
    size_t h = std::hash<const void*>()(k.base);
    h = h * 1000003u ^ (size_t)k.a; h = h * 1000003u ^ (size_t)k.b; h = h * 1000003u ^ (size_t)k.c; h = h * 1000003u ^ (size_t)k.kind;
    return h;
  }
};
static std::unordered_map<LpMapKey, CUtensorMap, LpMapKeyHash> g_lp_maps;
static std::mutex g_lp_mu;

// Rows of `cols` entries, `ld` apart: boxes of 64 entries x 64 rows.
static bool lp_rows_map(CUtensorMap* out, const void* base, long long rows, int cols, long long ld) {
  LpMapKey key{base, rows, cols, ld, 0};
  std::lock_guard<std::mutex> g(g_lp_mu);
  auto it = g_lp_maps.find(key);
  if (it != g_lp_maps.end()) { *out = it->second; return true; }
  TaEncodeFn fn = ta_encode_fn();
  if (!fn) return false;
  cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
  cuuint32_t box[2] = {64, TA_KEYS};
  cuuint32_t estr[2] = {1, 1};
  if (fn(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return false;
  if (g_lp_maps.size() > 4096) g_lp_maps.clear();
  g_lp_maps.emplace(key, *out);
  return true;
}

// `cols` entries of every head of queries [tokens, heads, head_size]: boxes of 64 entries x 1 head x 128 tokens; zeros behind `cols`.
static bool lp_q_map(CUtensorMap* out, const void* base, long long tokens, int heads, int head_size, int cols) {
  LpMapKey key{base, tokens, ((long long)heads << 32) | (unsigned)head_size, cols, 1};
  std::lock_guard<std::mutex> g(g_lp_mu);
  auto it = g_lp_maps.find(key);
  if (it != g_lp_maps.end()) { *out = it->second; return true; }
  TaEncodeFn fn = ta_encode_fn();
  if (!fn) return false;
  cuuint64_t dims[3] = {(cuuint64_t)cols, (cuuint64_t)heads, (cuuint64_t)tokens};
  cuuint64_t strides[2] = {(cuuint64_t)head_size * 2, (cuuint64_t)heads * head_size * 2};
  cuuint32_t box[3] = {64, 1, TA_ROWS};
  cuuint32_t estr[3] = {1, 1, 1};
  if (fn(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return false;
  if (g_lp_maps.size() > 4096) g_lp_maps.clear();
  g_lp_maps.emplace(key, *out);
  return true;
}

}  // namespace lb

// 1 when lb_latent_prefill takes these sizes.
LB_EXPORT int lb_latent_prefill_ok(int dim, int rot, int vdim, int kv_rank) {
  return dim > 0 && dim <= 128 && dim % 8 == 0 && rot >= 0 && rot <= 64 && rot % 8 == 0 && vdim > 0 && vdim <= 128 && vdim % 8 == 0 &&
         kv_rank > 0 && kv_rank % 8 == 0;
}

// out [total_rows, dk] (bfloat16, dk a multiple of 8) = the cached vectors of the requests in `entries` {request, first row, rows, unused},
// one row a position from 0 on, zeros behind a request's last position; the entries' rows lie one behind the other.
LB_EXPORT int lb_latent_gather(void* out, const void* pool, const void* entries, int num_entries, int total_rows, const int* context_lens,
                               const int* block_table, int max_pages, int page_size, int dk, cudaStream_t stream) {
  LB_CHECK_ARG(out && pool && entries && context_lens && block_table && num_entries >= 0 && total_rows >= 0 && max_pages > 0 && page_size > 0,
               "latent_gather: bad arguments");
  LB_CHECK_ARG(dk > 0 && dk % 8 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)pool % 16 == 0 && (uintptr_t)entries % 16 == 0,
               "latent_gather: vectors of %d entries must be whole 16-byte words", dk);
  if (total_rows == 0) return 0;
  lb::launch(lb::latent_gather_kernel, dim3((total_rows + 7) / 8), dim3(256), 0, stream, (uint4*)out, (const uint4*)pool, (const int4*)entries,
             num_entries, total_rows, context_lens, block_table, max_pages, page_size, dk / 8);
  LB_CHECK_LAUNCH("latent_gather");
  return 0;
}

// q [T, heads, dim + rot], out [T, heads, vdim], kv [rows, heads * (dim + vdim)] (all keys, then all values), lat [rows, kv_rank + rot], all
// bfloat16.  tiles: {first token, tokens <= 256, unused, first row of the request in kv and lat}; position j of the request is
// row first + j.  gate: optional float32 [T, heads], rows ldg apart.  key_splits > 1 (at most 8): ranges of keys through
// `workspace` (float32, tiles * heads * key_splits * 256 * (vdim + 2)).
LB_EXPORT int lb_latent_prefill(const void* q, void* out, const void* kv, const void* lat, const int* positions, const void* tiles, int num_tiles,
                                int num_tokens, int rows, int heads, int dim, int rot, int vdim, int kv_rank, float scale, const float* sinks,
                                const float* gate, long long ldg, int key_splits, float* workspace, long long workspace_elems, cudaStream_t stream) {
  LB_CHECK_ARG(lb_latent_prefill_ok(dim, rot, vdim, kv_rank) && heads > 0, "latent_prefill: heads of %d + %d (values %d) on a latent of %d are not taken", dim, rot,
               vdim, kv_rank);
  LB_CHECK_ARG(q && out && kv && lat && positions && tiles && num_tiles >= 0 && num_tokens > 0 && rows > 0 && scale > 0.f, "latent_prefill: bad arguments");
  LB_CHECK_ARG(((uintptr_t)q % 16 == 0) && ((uintptr_t)out % 16 == 0) && ((uintptr_t)kv % 16 == 0) && ((uintptr_t)lat % 16 == 0),
               "latent_prefill: operands must be 16-byte aligned");
  LB_CHECK_ARG(num_tiles <= 65535 && key_splits >= 1 && key_splits <= lb::LP_MAX_SPLITS, "latent_prefill: %d tiles, %d key ranges", num_tiles, key_splits);
  LB_CHECK_ARG(key_splits == 1 || (workspace && (uintptr_t)workspace % 16 == 0 &&
                                   workspace_elems >= (long long)num_tiles * heads * key_splits * lb::TA_PART_ROWS * (vdim + 2)),
               "latent_prefill: the workspace is too small");
  if (num_tiles == 0) return 0;
  CUtensorMap mqu, mqr, mkv, mlat;
  const int hd = dim + rot;
  bool ok = lb::lp_q_map(&mqu, q, num_tokens, heads, hd, dim) && lb::lp_rows_map(&mkv, kv, rows, heads * (dim + vdim), (long long)heads * (dim + vdim)) &&
            lb::lp_rows_map(&mlat, lat, rows, kv_rank + rot, kv_rank + rot);
  if (ok) ok = rot > 0 ? lb::lp_q_map(&mqr, (const lb::bf16*)q + dim, num_tokens, heads, hd, rot) : lb::lp_q_map(&mqr, q, num_tokens, heads, hd, dim);
  if (!ok) { lb::set_error("latent_prefill: cuTensorMapEncodeTiled failed"); return 3; }
  lb::LatentPrefillParams p;
  p.out = (lb::bf16*)out; p.positions = positions; p.tiles = (const int4*)tiles; p.sinks = sinks; p.gate = gate; p.ldg = ldg;
  p.heads = heads; p.dim = dim; p.rot = rot; p.vdim = vdim; p.kv_rank = kv_rank; p.dim_chunks = (dim + 63) / 64;
  p.chunks = p.dim_chunks + (rot > 0 ? 1 : 0); p.scale_log2 = scale * 1.4426950408889634f;
  p.part_o = workspace;
  p.part_ml = key_splits > 1 ? workspace + (size_t)num_tiles * heads * key_splits * lb::TA_PART_ROWS * vdim : nullptr;
  const int smem = lb::LP_SMEM_BYTES + 1024;
  static_assert(lb::LP_SMEM_BYTES + 1024 <= 232448, "a CTA has 227 KB of shared memory");
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(lb::latent_prefill_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(lb::latent_prefill_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) { lb::set_error("latent_prefill: cannot reserve %d bytes of shared memory: %s", smem, cudaGetErrorString(e)); return 2; }
    configured = true;
  }
  const dim3 grid(heads, num_tiles, key_splits);
  if (vdim <= 64) lb::launch(lb::latent_prefill_kernel<1>, grid, dim3(lb::LP_THREADS), smem, stream, mqu, mqr, mkv, mlat, p);
  else lb::launch(lb::latent_prefill_kernel<2>, grid, dim3(lb::LP_THREADS), smem, stream, mqu, mqr, mkv, mlat, p);
  LB_CHECK_LAUNCH("latent_prefill");
  if (key_splits > 1) {
    lb::launch(lb::latent_prefill_combine_kernel, dim3(num_tiles, heads, lb::TA_PART_ROWS / 8), dim3(32, 8), 0, stream, p, key_splits);
    LB_CHECK_LAUNCH("latent_prefill combine");
  }
  return 0;
}

// Reads and clears the flag a bounded wait of this kernel sets when it gives up (0: none).
LB_EXPORT int lb_latent_prefill_device_error() {
  int v = 0, zero = 0;
  if (cudaMemcpyFromSymbol(&v, lb::g_attention_tc_error, sizeof(int)) != cudaSuccess) return -1;
  if (v != 0) cudaMemcpyToSymbol(lb::g_attention_tc_error, &zero, sizeof(int));
  return v;
}
