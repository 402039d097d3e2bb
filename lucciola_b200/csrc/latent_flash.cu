// Attention of many query heads over ONE cached vector a token that is key and value at once (bfloat16): the key is the whole
// vector of `dk` entries, the value its first `dv`.  That is latent attention with the heads' key maps moved to the queries and
// their value maps behind the sum: dk = latent + rotated part (512 + 64, say), dv = the latent.  Decoded tokens and
// portions of prompts; causal, with an optional sink a head (one more term exp(sink) of the denominator without a value).
//
// A work item ("tile") is a run of consecutive tokens of one request and a group of G heads whose G * tokens <= MT * 16
// query rows share every cached vector the CTA reads.  The keys of a tile may be cut into `splits` ranges (grid z) whose
// unnormalised results (m, l, o) a second kernel adds up in the ranges' order.
//
// Per CTA a ninth warp fetches: stages of 64 cached vectors by TMA, in groups of eight: one box brings all entries of a group's
// vectors, as chunks of 64 entries x 8 vectors in the 128-byte swizzle (a CTA can issue a box in some hundred cycles
// whatever its size, so few large ones; sizes that are no multiple of 64 take a box a chunk, which reads zeros past dk).  The eight computing warps work on a stage in two phases:
//     S = Q K^T    the MT row blocks of 16 times the 64 keys are shared out (MT = 1: 8 keys a warp, 2: one row block and 16
//                  keys, 4: one row block and 32 keys); maxima meet through shared memory; P goes there in bfloat16
//     O += P V     each warp owns an eighth of the value entries for ALL rows, so the values are read once from shared
//                  memory and the sums of a tile (64 rows x 512 entries in 32-bit) lie spread over the CTA's registers
// The softmax is the online form (m, l, o per row, 32-bit).  Rows of the last stage that hold no key of the sequence are set
// to zero before they are read, so that nothing a reused page holds can reach a sum.
#include "warp_mma.cuh"

#include <cuda.h>
#include <mutex>
#include <unordered_map>

namespace lb {

constexpr int LF_KEYS = 64;                   // cached vectors of a stage
constexpr int LF_WARPS = 8;                   // computing warps
constexpr int LF_THREADS = (LF_WARPS + 1) * 32;
constexpr int LF_CHUNK = LF_KEYS * 128;       // 64 entries of 64 vectors: 8 KB
enum { LF_ERR_FULL = 501, LF_ERR_EMPTY = 502 };
__device__ int g_latent_flash_error = 0;

struct LatentFlashParams {
  const bf16* q; bf16* out;                   // [T, heads, dk], [T, heads, dv]
  const int* positions;
  const int* block_table; int max_pages;
  const int4* tiles;                          // {first token, tokens, request index, the request's tokens in this step before the first}
  const float* sinks;                         // optional [heads]
  float* part_o; float* part_ml;              // [tiles, head groups, splits, part_rows, dv | 2]
  int part_rows, splits;
  int heads, group, dk, dv, page_size, page_shift;
  float scale_log2;                           // scale * log2(e)
  int whole;                                  // 1: a box brings whole vectors (dk a multiple of 64)
};

__device__ __forceinline__ void lf_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
__device__ __forceinline__ void lf_tma_3d(uint32_t dst, const CUtensorMap* map, int x, int y, int z, uint32_t bar) {
  asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];"
               ::"r"(dst), "l"(map), "r"(x), "r"(y), "r"(z), "r"(bar) : "memory");
}
// Byte offset of 16-byte piece c (over the whole vector) of vector r in a stage: groups of eight vectors, chunks of 64 entries.
template <int NK>
__device__ __forceinline__ uint32_t lf_stage_offset(int r, int c) {
  return (uint32_t)((r >> 3) * (NK * 1024) + (c >> 3) * 1024 + (r & 7) * 128 + (((c & 7) ^ (r & 7)) << 4));
}
// Byte offset of 16-byte piece c (over the whole row) of row r in a matrix of `rows` rows cut into chunks of 64 entries.
__device__ __forceinline__ uint32_t lf_offset(int rows, int r, int c) {
  return (uint32_t)((c >> 3) * rows * 128 + r * 128 + (((c & 7) ^ (r & 7)) << 4));
}

__host__ __device__ constexpr int lf_stages(int nk) { return nk >= 8 ? 2 : (nk >= 5 ? 3 : 4); }
__host__ __device__ constexpr int lf_smem_bytes(int nk, int mt) {
  return 1024 + lf_stages(nk) * nk * LF_CHUNK + mt * 16 * nk * 128 + mt * 16 * 128 + (8 / mt) * mt * 16 * 4 + 2 * mt * 16 * 4;
}

// NK, NV: chunks of 64 entries of a key and of a value; MT: row blocks of 16.
template <int NK, int NV, int MT>
__global__ void __launch_bounds__(LF_THREADS, 1)
latent_flash_kernel(const __grid_constant__ CUtensorMap kmap, LatentFlashParams p) {
  constexpr int STAGES = lf_stages(NK);
  constexpr int STAGE_BYTES = NK * LF_CHUNK;
  constexpr int ROWS = MT * 16;
  constexpr int KSPLIT = LF_WARPS / MT;         // warps that share a row block's keys
  constexpr int KPW = LF_KEYS / KSPLIT;         // keys of a warp in the first phase: 8, 16 or 32
  constexpr int NB = KPW / 8;
  constexpr int VPW = NV * 64 / LF_WARPS;       // value entries of a warp in the second phase
  constexpr int ND = VPW / 8;
  static_assert(ND % 2 == 0, "a warp's value entries come in sixteens");
  extern __shared__ uint8_t lf_smem_raw[];
  __shared__ __align__(8) unsigned long long bars[2 * STAGES];
  __shared__ int abort_word[2];                 // the computing warps' and the fetching warp's
  volatile int* abort_flag = &abort_word[0];
  const uint32_t base = ((uint32_t)__cvta_generic_to_shared(lf_smem_raw) + 1023u) & ~1023u;
  uint8_t* base_ptr = lf_smem_raw + (base - (uint32_t)__cvta_generic_to_shared(lf_smem_raw));
  const uint32_t q_smem = base + STAGES * STAGE_BYTES, p_smem = q_smem + ROWS * NK * 128;
  float* red = reinterpret_cast<float*>(base_ptr + STAGES * STAGE_BYTES + ROWS * NK * 128 + ROWS * 128);    // [KSPLIT][ROWS]
  float* alpha_s = red + KSPLIT * ROWS;                                                                   // [ROWS]
  float* m_s = alpha_s + ROWS;                                                                            // [ROWS]
  auto full = [&](int s) { return (uint32_t)__cvta_generic_to_shared(&bars[s]); };
  auto empty = [&](int s) { return (uint32_t)__cvta_generic_to_shared(&bars[STAGES + s]); };

  pdl_trigger();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int4 tile = p.tiles[blockIdx.x];
  const int t0 = tile.x, ntok = tile.y, seq = tile.z;
  const int hg = blockIdx.y, split = blockIdx.z;
  const int G = p.group, rows = ntok * G;
  const int pos0 = p.positions[t0];
  const int* bt = p.block_table + (size_t)seq * p.max_pages;
  const int span = pos0 + ntok;
  const int per_split = ((span + p.splits - 1) / p.splits + LF_KEYS - 1) / LF_KEYS * LF_KEYS;
  const int kbeg = split * per_split;
  const int kend = min(span, kbeg + per_split);              // exclusive
  const int num_stages = kend > kbeg ? (kend - kbeg + LF_KEYS - 1) / LF_KEYS : 0;

  if (tid == 0) {
    for (int s = 0; s < STAGES; ++s) { mbar_init(full(s), 1); mbar_init(empty(s), LF_WARPS); }
    abort_word[0] = abort_word[1] = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();

  if (warp == LF_WARPS) {
    // ---- the fetching warp ------------------------------------------------------------------------------------------------
    const int pieces = p.whole ? 1 : NK;                       // boxes of a group of eight vectors
    auto fetch = [&](int st) {
      const int b = st % STAGES;
      if (lane == 0) mbar_expect_tx(full(b), STAGE_BYTES);
      __syncwarp();
      for (int op = lane; op < 8 * pieces; op += 32) {
        const int group = op / pieces, chunk = op - group * pieces;
        const int key0 = kbeg + st * LF_KEYS + group * 8;
        const int page = key0 < kend ? bt[key0 >> p.page_shift] : -1;
        const int row = page >= 0 ? page * p.page_size + (key0 & (p.page_size - 1)) : 0;      // page 0 where there is none: cleared below
        const uint32_t dst = base + b * STAGE_BYTES + group * (NK * 1024) + chunk * 1024;
        if (p.whole) lf_tma_3d(dst, &kmap, 0, row, 0, full(b));
        else lf_tma_3d(dst, &kmap, chunk * 64, row, 0, full(b));
      }
    };
    // Vectors before the request's first token of this step were written by earlier steps: the first stages of them are requested while
    // the kernel ahead (which writes this step's) may still run.
    int st = 0;
    for (; st < min(num_stages, STAGES) && kbeg + (st + 1) * LF_KEYS <= pos0 - tile.w; ++st) fetch(st);
    pdl_wait();
    for (; st < num_stages; ++st) {
      if (!mbar_wait<true>(empty(st % STAGES), (uint32_t)((st / STAGES) & 1) ^ 1u, &abort_word[1], &g_latent_flash_error, LF_ERR_EMPTY)) break;
      fetch(st);
    }
    // nobody leaves while a copy of its own is in flight
    for (int j = max(0, st - STAGES); j < st; ++j)
      mbar_wait<true>(full(j % STAGES), (uint32_t)((j / STAGES) & 1), &abort_word[1], &g_latent_flash_error, LF_ERR_FULL);
    return;
  }

  // ---- the computing warps --------------------------------------------------------------------------------------------------
  const bool hole = num_stages > 0 && bt[kbeg >> p.page_shift] < 0;      // an entry that owns no page (padding of a recorded step)
  pdl_wait();
  for (int idx = tid; idx < ROWS * NK * 8; idx += LF_WARPS * 32) {
    const int r = idx / (NK * 8), c = idx % (NK * 8);
    const bool valid = r < rows && c * 8 < p.dk;
    const bf16* src = p.q;
    if (valid) src = p.q + ((size_t)(t0 + r / G) * p.heads + hg * G + r % G) * p.dk + c * 8;
    cp_async16(q_smem + lf_offset(ROWS, r, c), src, valid);
  }
  cp_async_commit();

  const int wm = warp / KSPLIT, wn = warp % KSPLIT;          // first phase: row block, share of the keys
  const int r0 = wm * 16 + (lane >> 2);
  int row_pos[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) row_pos[h] = r0 + 8 * h < rows ? pos0 + (r0 + 8 * h) / G : -1;      // -1: no key passes the mask
  const int v_col = warp * (VPW / 8);                        // second phase: first 16-byte piece of this warp's value entries

  float o[MT][ND][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < ND; ++i) { o[mt][i][0] = o[mt][i][1] = o[mt][i][2] = o[mt][i][3] = 0.f; }
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  cp_async_wait<0>();
  lf_sync();

  for (int st = 0; st < num_stages; ++st) {
    const int b = st % STAGES;
    const uint32_t kb = base + b * STAGE_BYTES;
    const int kbase = kbeg + st * LF_KEYS;
    mbar_wait<false>(full(b), (uint32_t)((st / STAGES) & 1), abort_flag, &g_latent_flash_error, LF_ERR_FULL);
    // A wait that gave up leaves its mark; the warps read it behind the next barrier and leave together.
    if (kbase + LF_KEYS > kend || hole) {                    // uniform over the CTA
      const int first = hole ? 0 : kend - kbase;
      for (int idx = tid; idx < (LF_KEYS - first) * NK * 8; idx += LF_WARPS * 32)
        asm volatile("st.shared.v4.b32 [%0], {%1, %1, %1, %1};" ::"r"(kb + lf_stage_offset<NK>(first + idx / (NK * 8), idx % (NK * 8))), "r"(0) : "memory");
      lf_sync();
    }

    // ---- S = Q K^T: this warp's 16 rows x KPW keys -----------------------------------------------------------------------
    float s[NB][4];
#pragma unroll
    for (int i = 0; i < NB; ++i) { s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f; }
    const int a_row = wm * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
    if (NB == 1) {
#pragma unroll 6
      for (int kk = 0; kk < NK * 4; kk += 2) {
        uint32_t a[2][4], b0, b1, b2, b3;
        ldmatrix_x4(q_smem + lf_offset(ROWS, a_row, kk * 2 + (lane >> 4)), a[0][0], a[0][1], a[0][2], a[0][3]);
        ldmatrix_x4(q_smem + lf_offset(ROWS, a_row, kk * 2 + 2 + (lane >> 4)), a[1][0], a[1][1], a[1][2], a[1][3]);
        // matrices: the four 16-byte pieces of two steps
        ldmatrix_x4(kb + lf_stage_offset<NK>(wn * KPW + (lane & 7), kk * 2 + (lane >> 3)), b0, b1, b2, b3);
        mma_bf16(s[0], a[0], b0, b1);
        mma_bf16(s[0], a[1], b2, b3);
      }
    } else {
#pragma unroll 6
      for (int kk = 0; kk < NK * 4; ++kk) {
        uint32_t a[4];
        ldmatrix_x4(q_smem + lf_offset(ROWS, a_row, kk * 2 + (lane >> 4)), a[0], a[1], a[2], a[3]);
#pragma unroll
        for (int nb = 0; nb + 1 < NB; nb += 2) {
          // matrices: (keys nb, lo), (keys nb, hi), (keys nb + 1, lo), (keys nb + 1, hi)
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(kb + lf_stage_offset<NK>(wn * KPW + nb * 8 + (lane & 7) + (lane >> 4) * 8, kk * 2 + ((lane >> 3) & 1)), b0, b1, b2, b3);
          mma_bf16(s[nb], a, b0, b1);
          mma_bf16(s[nb + 1 < NB ? nb + 1 : nb], a, b2, b3);
        }
      }
    }

    // ---- mask, maxima over the warps that share the rows ------------------------------------------------------------------
    const bool need_mask = kbase + LF_KEYS - 1 > pos0 || kbase + LF_KEYS > kend;
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nb = 0; nb < NB; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int h = e >> 1;
        if (need_mask) {
          const int j = kbase + wn * KPW + nb * 8 + (lane & 3) * 2 + (e & 1);
          if (j > row_pos[h] || j >= kend) s[nb][e] = -INFINITY;
        }
        mx[h] = fmaxf(mx[h], s[nb][e]);
      }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
      mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
      if ((lane & 3) == 0) red[wn * ROWS + r0 + 8 * h] = mx[h];
    }
    lf_sync();
    if (*abort_flag) break;
    float m_use[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float m_new = m_run[h];
#pragma unroll
      for (int z = 0; z < KSPLIT; ++z) m_new = fmaxf(m_new, red[z * ROWS + r0 + 8 * h]);
      m_use[h] = m_new == -INFINITY ? 0.f : m_new * p.scale_log2;
      const float alpha = m_run[h] == -INFINITY ? 0.f : exp2f(m_run[h] * p.scale_log2 - m_use[h]);
      m_run[h] = m_new;
      l_run[h] *= alpha;
      if (wn == 0 && (lane & 3) == 0) alpha_s[r0 + 8 * h] = alpha;
    }
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) {
      const int key = wn * KPW + nb * 8 + (lane & 3) * 2;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const float p0 = exp2_approx(fmaf(s[nb][2 * h], p.scale_log2, -m_use[h]));        // 2^-inf = 0 for masked keys
        const float p1 = exp2_approx(fmaf(s[nb][2 * h + 1], p.scale_log2, -m_use[h]));
        l_run[h] += p0 + p1;
        asm volatile("st.shared.b32 [%0], %1;" ::"r"(p_smem + lf_offset(ROWS, r0 + 8 * h, key >> 3) + (key & 7) * 2), "r"(pack_bf16(p0, p1)) : "memory");
      }
    }
    lf_sync();

    // ---- O += P V: all rows x this warp's value entries --------------------------------------------------------------------
    float al[MT][2];
    bool same = true;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        al[mt][h] = alpha_s[mt * 16 + (lane >> 2) + 8 * h];
        same = same && al[mt][h] == 1.f;
      }
    // Once the maxima have settled the factors are exactly 1 for stage after stage: skip the multiplications then.
    if (!__all_sync(0xffffffffu, same)) {
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int i = 0; i < ND; ++i) { o[mt][i][0] *= al[mt][0]; o[mt][i][1] *= al[mt][0]; o[mt][i][2] *= al[mt][1]; o[mt][i][3] *= al[mt][1]; }
    }
#pragma unroll
    for (int ks = 0; ks < LF_KEYS / 16; ++ks) {
      uint32_t a[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
        ldmatrix_x4(p_smem + lf_offset(ROWS, mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, ks * 2 + (lane >> 4)), a[mt][0], a[mt][1], a[mt][2], a[mt][3]);
#pragma unroll
      for (int db = 0; db < ND; db += 2) {
        // matrices (transposed on load): (keys lo, entries db), (keys hi, db), (keys lo, db + 1), (keys hi, db + 1)
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(kb + lf_stage_offset<NK>(ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, v_col + db + (lane >> 4)), b0, b1, b2, b3);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_bf16(o[mt][db], a[mt], b0, b1);
          mma_bf16(o[mt][db + 1], a[mt], b2, b3);
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(empty(b));          // this warp has read the stage
  }

  // ---- sums of the rows over the warps that shared them, then out -----------------------------------------------------------
  lf_sync();
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
    l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
    if ((lane & 3) == 0) {
      red[wn * ROWS + r0 + 8 * h] = l_run[h];
      if (wn == 0) m_s[r0 + 8 * h] = m_run[h] == -INFINITY ? -INFINITY : m_run[h] * p.scale_log2;
    }
  }
  lf_sync();
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = mt * 16 + (lane >> 2) + 8 * h;
      if (r >= rows) continue;
      float L = 0.f;
#pragma unroll
      for (int z = 0; z < KSPLIT; ++z) L += red[z * ROWS + r];
      const float M = m_s[r];
      const int head = hg * G + r % G;
      if (p.splits == 1) {
        float f = 1.f, den = L;
        if (p.sinks) {
          const float sink = p.sinks[head] * 1.4426950408889634f, top = fmaxf(M, sink);
          f = M == -INFINITY ? 0.f : exp2f(M - top);
          den = L * f + exp2f(sink - top);
        }
        f = den > 0.f ? f / den : 0.f;
        bf16* dst = p.out + ((size_t)(t0 + r / G) * p.heads + head) * p.dv;
#pragma unroll
        for (int i = 0; i < ND; ++i) {
          const int e = (v_col + i) * 8 + (lane & 3) * 2;
          if (e < p.dv) *reinterpret_cast<__nv_bfloat162*>(dst + e) = __floats2bfloat162_rn(o[mt][i][2 * h] * f, o[mt][i][2 * h + 1] * f);
        }
      } else {
        const size_t slot = (((size_t)blockIdx.x * gridDim.y + hg) * p.splits + split) * p.part_rows + r;
        if (num_stages > 0) {                          // a range without keys leaves (-inf, 0) and no sums
          float* dst = p.part_o + slot * p.dv;
#pragma unroll
          for (int i = 0; i < ND; ++i) {
            const int e = (v_col + i) * 8 + (lane & 3) * 2;
            if (e < p.dv) *reinterpret_cast<float2*>(dst + e) = make_float2(o[mt][i][2 * h], o[mt][i][2 * h + 1]);
          }
        }
        if (warp == 0 && (lane & 3) == 0) { p.part_ml[slot * 2] = M; p.part_ml[slot * 2 + 1] = L; }
      }
    }
}

// out = sum_z 2^(m_z - M) o_z / (sum_z 2^(m_z - M) l_z + 2^(sink - M)), the ranges in their order.  One CTA a row.
constexpr int LF_MAX_SPLITS = 64;
__global__ void __launch_bounds__(128) latent_flash_combine_kernel(LatentFlashParams p) {
  __shared__ float wz[LF_MAX_SPLITS];
  __shared__ float den_s;
  pdl_trigger();
  const int4 tile = p.tiles[blockIdx.y];
  const int hg = blockIdx.z, r = blockIdx.x, G = p.group;
  if (r >= tile.y * G) return;
  const int head = hg * G + r % G;
  const float sink = p.sinks ? p.sinks[head] * 1.4426950408889634f : -INFINITY;
  pdl_wait();
  const size_t base = ((size_t)blockIdx.y * gridDim.z + hg) * p.splits;
  if (threadIdx.x < 32) {                      // the ranges' weights: a lane two of them
    float2 ml[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int z = threadIdx.x + 32 * u;
      ml[u] = z < p.splits ? *reinterpret_cast<const float2*>(p.part_ml + ((base + z) * p.part_rows + r) * 2) : make_float2(-INFINITY, 0.f);
    }
    const float M = fmaxf(sink, warp_max(fmaxf(ml[0].x, ml[1].x)));
    float den = 0.f;
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const float w = ml[u].x == -INFINITY ? 0.f : exp2f(ml[u].x - M);
      wz[threadIdx.x + 32 * u] = w;
      den += ml[u].y * w;
    }
    den = warp_sum(den) + (sink == -INFINITY ? 0.f : exp2f(sink - M));
    if (threadIdx.x == 0) den_s = den;
  }
  __syncthreads();
  const float inv = den_s > 0.f ? 1.f / den_s : 0.f;
  bf16* dst = p.out + ((size_t)(tile.x + r / G) * p.heads + head) * p.dv;
  for (int e = threadIdx.x * 4; e < p.dv; e += blockDim.x * 4) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int z0 = 0; z0 < p.splits; z0 += 8) {
      float4 a[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const bool have = z0 + u < p.splits && wz[z0 + u] != 0.f;        // what weighs nothing may never have been written
        a[u] = have ? *reinterpret_cast<const float4*>(p.part_o + ((base + z0 + u) * p.part_rows + r) * p.dv + e) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int u = 0; u < 8; ++u)
        if (z0 + u < p.splits) {
          const float w = wz[z0 + u];
          acc.x = fmaf(w, a[u].x, acc.x); acc.y = fmaf(w, a[u].y, acc.y); acc.z = fmaf(w, a[u].z, acc.z); acc.w = fmaf(w, a[u].w, acc.w);
        }
    }
    __nv_bfloat162 lo = __floats2bfloat162_rn(acc.x * inv, acc.y * inv), hi = __floats2bfloat162_rn(acc.z * inv, acc.w * inv);
    *reinterpret_cast<uint2*>(dst + e) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
  }
}

// ---- host side ---------------------------------------------------------------------------------------------------------------
typedef CUresult (*LfEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                               const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                               CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
struct LfMapKey {
  const void* base; long long rows; int d, box;             // box: chunks of a box
  bool operator==(const LfMapKey& o) const { return base == o.base && rows == o.rows && d == o.d && box == o.box; }
};
struct LfMapKeyHash {
  size_t operator()(const LfMapKey& k) const {
    size_t h = std::hash<const void*>()(k.base);
    h = h * 1000003u ^ (size_t)k.rows; h = h * 1000003u ^ (size_t)k.d; h = h * 1000003u ^ (size_t)k.box;
    return h;
  }
};
static std::unordered_map<LfMapKey, CUtensorMap, LfMapKeyHash> g_lf_maps;
static std::mutex g_lf_mu;

// A pool [pages, page size, d] as rows of d entries: boxes of 8 rows x 64 entries, and with chunks > 0 (d a multiple of 64) so many
// chunks of 64 entries one behind the other; what lies past d reads as zeros.
static bool lf_pool_map(CUtensorMap* out, const void* pool, long long rows, int d, int box) {
  LfMapKey key{pool, rows, d, box};
  std::lock_guard<std::mutex> g(g_lf_mu);
  auto it = g_lf_maps.find(key);
  if (it != g_lf_maps.end()) { *out = it->second; return true; }
  void* sym = nullptr;
  cudaDriverEntryPointQueryResult q;
  if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) return false;
  cuuint64_t dims[3] = {(cuuint64_t)(box > 0 ? 64 : d), (cuuint64_t)rows, (cuuint64_t)(box > 0 ? d / 64 : 1)};
  cuuint64_t strides[2] = {(cuuint64_t)d * 2, 128};
  cuuint32_t bx[3] = {64, 8, (cuuint32_t)(box > 0 ? box : 1)};
  cuuint32_t estr[3] = {1, 1, 1};
  if (((LfEncodeFn)sym)(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(pool), dims, strides, bx, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                        CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return false;
  if (g_lf_maps.size() > 4096) g_lf_maps.clear();
  g_lf_maps.emplace(key, *out);
  return true;
}

template <int NK, int NV, int MT>
static cudaError_t lf_launch(const CUtensorMap& map, const LatentFlashParams& p, int num_tiles, int head_groups, cudaStream_t stream) {
  static bool configured = false;
  constexpr int smem = lf_smem_bytes(NK, MT);
  static_assert(smem <= 232448, "a CTA has 227 KB of shared memory");
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(latent_flash_kernel<NK, NV, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  launch(latent_flash_kernel<NK, NV, MT>, dim3(num_tiles, head_groups, p.splits), dim3(LF_THREADS), smem, stream, map, p);
  return cudaSuccess;
}

}  // namespace lb

// 1 when lb_latent_flash takes these sizes.
LB_EXPORT int lb_latent_flash_ok(int dk, int dv, int group, int page_size) {
  if (dk % 8 || dv % 8 || dv <= 0 || dv > dk || dk > 576 || dv > 512 || group < 1 || group > 64) return 0;
  if (page_size < 8 || page_size > 128 || (page_size & (page_size - 1))) return 0;
  return 1;
}

// Reads and clears the flag a bounded wait of this kernel sets when it gives up (0: none).
LB_EXPORT int lb_latent_flash_device_error() {
  int v = 0, zero = 0;
  if (cudaMemcpyFromSymbol(&v, lb::g_latent_flash_error, sizeof(int)) != cudaSuccess) return -1;
  if (v != 0) cudaMemcpyToSymbol(lb::g_latent_flash_error, &zero, sizeof(int));
  return v;
}

// q [T, heads, dk], out [T, heads, dv], pool [pages, 1, page_size, dk], all bfloat16.  tiles: {first token, tokens, request
// index, the request's tokens in this step before the tile's first}, tokens * group <= part_rows <= 64; `group` heads (a divisor of heads) share a tile.  splits > 1 (at most 64):
// the keys of a tile in that many ranges, added up through `workspace` (float32, tiles * heads / group * splits * part_rows * (dv + 2)).
LB_EXPORT int lb_latent_flash(const void* q, void* out, const void* pool, const int* positions, const int* block_table, const void* tiles,
                              int num_tiles, int heads, int group, int dk, int dv, int page_size, int max_pages, int num_pages,
                              float scale, const float* sinks, int splits, int part_rows, float* workspace, long long workspace_elems,
                              cudaStream_t stream) {
  LB_CHECK_ARG(lb_latent_flash_ok(dk, dv, group, page_size) && heads > 0 && heads % group == 0,
               "latent_flash: keys of %d (values %d) in pages of %d for groups of %d of %d heads are not taken", dk, dv, page_size, group, heads);
  LB_CHECK_ARG(scale > 0.f && max_pages > 0 && num_pages > 0 && num_tiles >= 0 && part_rows >= group && part_rows <= 64, "latent_flash: bad arguments");
  LB_CHECK_ARG(((uintptr_t)q % 16 == 0) && ((uintptr_t)out % 16 == 0) && ((uintptr_t)pool % 16 == 0), "latent_flash: operands must be 16-byte aligned");
  const int hgroups = heads / group;
  LB_CHECK_ARG(splits >= 1 && splits <= lb::LF_MAX_SPLITS, "latent_flash: %d key ranges", splits);
  LB_CHECK_ARG(splits == 1 || (workspace && (uintptr_t)workspace % 16 == 0 &&
                               workspace_elems >= (long long)num_tiles * hgroups * splits * part_rows * (dv + 2)), "latent_flash: the workspace is too small");
  LB_CHECK_ARG(num_tiles <= 65535 && hgroups <= 65535, "latent_flash: too many tiles");
  if (num_tiles == 0) return 0;
  CUtensorMap map;
  const int nk = (dk + 63) / 64, nv = (dv + 63) / 64;
  const int nk_padded = nk <= 2 ? 2 : (nk <= 3 && nv <= 2) ? 3 : (nk <= 5 && nv <= 4) ? 5 : 9;
  if (!lb::lf_pool_map(&map, pool, (long long)num_pages * page_size, dk, dk % 64 == 0 ? nk_padded : 0)) {
    lb::set_error("latent_flash: cuTensorMapEncodeTiled failed");
    return 3;
  }
  lb::LatentFlashParams p;
  p.q = (const lb::bf16*)q; p.out = (lb::bf16*)out; p.positions = positions; p.block_table = block_table; p.max_pages = max_pages;
  p.tiles = (const int4*)tiles; p.sinks = sinks; p.part_rows = part_rows; p.splits = splits; p.heads = heads; p.group = group;
  p.dk = dk; p.dv = dv; p.page_size = page_size; p.scale_log2 = scale * 1.4426950408889634f; p.whole = dk % 64 == 0 ? 1 : 0;
  p.part_o = workspace;
  p.part_ml = splits > 1 ? workspace + (size_t)num_tiles * hgroups * splits * part_rows * dv : nullptr;
  p.page_shift = 0;
  while ((1 << p.page_shift) < page_size) ++p.page_shift;
  const int mt = part_rows <= 16 ? 1 : (part_rows <= 32 ? 2 : 4);
  cudaError_t e;
#define LB_LF(NK, NV) \
  (mt == 1 ? lb::lf_launch<NK, NV, 1>(map, p, num_tiles, hgroups, stream) : mt == 2 ? lb::lf_launch<NK, NV, 2>(map, p, num_tiles, hgroups, stream) \
                                                                                   : lb::lf_launch<NK, NV, 4>(map, p, num_tiles, hgroups, stream))
  if (nk_padded == 2) e = LB_LF(2, 2);
  else if (nk_padded == 3) e = LB_LF(3, 2);
  else if (nk_padded == 5) e = LB_LF(5, 4);
  else e = LB_LF(9, 8);
#undef LB_LF
  if (e != cudaSuccess) { lb::set_error("latent_flash: cannot reserve shared memory: %s", cudaGetErrorString(e)); return 2; }
  LB_CHECK_LAUNCH("latent_flash");
  if (splits > 1) {
    lb::launch(lb::latent_flash_combine_kernel, dim3(part_rows, num_tiles, hgroups), dim3(128), 0, stream, p);
    LB_CHECK_LAUNCH("latent_flash combine");
  }
  return 0;
}
