// Per-head RMSNorm of q and k, rotary position encoding, and the write of the
// new keys and values into their pages: one launch for what lucciola runs as
// two norms (src/qwen.cc:617-632), two rotations (src/qwen.cc:635-644,
// src/kernels/rope.cu:28-60) and the cache append
// (src/kernels/attention_paged.cu:26-44).
//
// Order as in the reference: norm over the head (weight [d] shared by all
// heads), then the rotation of the pairs (i, i + rot/2) by pos * inv_freq[i]
// ("NeoX" halves), then the write.  v is copied unchanged.  All arithmetic is
// 32-bit; the angle is one 32-bit product of the position and a host-made
// table entry, so a plain implementation that uses the same table gets the
// same angle.
//
// Page layout of one cache layer: [page][kv_head][slot][d].
//
// Two more forms lucciola does not have.  `pairs`: the pairs are neighbours, (2i, 2i + 1), instead of (i, i + rot/2).
// `unit`: after the rotation every q and k head is divided by its root mean square (sqrt(mean(x^2) + eps), no weight).
// And a query temperature: behind all that the queries at position p are multiplied by 1 + coef * ln(floor((p + 1) / every) + 1).
#include "common.cuh"

#include <type_traits>

namespace lb {

struct RopeKvParams {
  const void* q_in; const void* k_in; const void* v_in;
  long long q_stride, k_stride, v_stride;   // elements between token rows
  void* q_out;                               // [T, nq, d]
  void* k_out; void* v_out;                  // optional [T, nkv, d] (when no cache is given)
  void* k_cache; void* v_cache;              // optional pools
  const int* positions; const int* token_seq; const int* block_table;
  const float* q_norm_w; const float* k_norm_w; const float* inv_freq;
  int num_q_heads, num_kv_heads, head_dim, rot_dim, page_size, max_pages;
  float eps;
  int v_dim;                                 // size of a value head (the value pool and v_out have rows of this size)
  float rot_scale;                           // sines and cosines are multiplied by this (1: a pure rotation)
  int pairs;                                 // 1: neighbours (2i, 2i + 1) are a pair, not (i, i + rot/2)
  int unit;                                  // 1: divided by the root mean square behind the rotation, without a weight
  float temp_coef; int temp_every;           // temp_every > 0: queries are multiplied by their position's temperature
};

// 1 + coef * ln(floor((p + 1) / every) + 1), or 1 without a temperature.
__device__ __forceinline__ float query_temperature(const RopeKvParams& p, int pos) {
  return p.temp_every > 0 ? 1.f + p.temp_coef * logf((float)((pos + 1) / p.temp_every + 1)) : 1.f;
}

// TI: the type of q_in, k_in, v_in (a product's output, which may be 32-bit where the heads are stored in bfloat16)
template <typename T, typename TI>
__global__ void rope_kv_kernel(RopeKvParams p) {
  extern __shared__ float smem[];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  const int d = p.head_dim, dv = p.v_dim, half = p.rot_dim >> 1;
  float* buf = smem + (size_t)warp * d;
  const int pos = p.positions[t];
  const float temp = query_temperature(p, pos);
  const int total_heads = p.num_q_heads + 2 * p.num_kv_heads;

  // One head per warp: the grid's second dimension covers the heads.
  for (int h = blockIdx.y * nwarps + warp; h < total_heads; h += gridDim.y * nwarps) {
    const int kind = h < p.num_q_heads ? 0 : (h < p.num_q_heads + p.num_kv_heads ? 1 : 2);
    const int hh = kind == 0 ? h : (kind == 1 ? h - p.num_q_heads : h - p.num_q_heads - p.num_kv_heads);
    const int dh = kind == 2 ? dv : d;        // this head's size
    const TI* src = kind == 0 ? (const TI*)p.q_in + (size_t)t * p.q_stride + (size_t)hh * d
                  : kind == 1 ? (const TI*)p.k_in + (size_t)t * p.k_stride + (size_t)hh * d
                              : (const TI*)p.v_in + (size_t)t * p.v_stride + (size_t)hh * dv;
    T* dst = nullptr;
    if (kind == 0) {
      dst = (T*)p.q_out + ((size_t)t * p.num_q_heads + hh) * d;
    } else if (p.k_cache) {
      const int seq = p.token_seq[t];
      const int page = p.block_table[(size_t)seq * p.max_pages + pos / p.page_size];
      const int slot = pos % p.page_size;
      if (page >= 0) {
        T* pool = (T*)(kind == 1 ? p.k_cache : p.v_cache);
        dst = pool + (((size_t)page * p.num_kv_heads + hh) * p.page_size + slot) * dh;
      }
    } else {
      T* o = (T*)(kind == 1 ? p.k_out : p.v_out);
      if (o) dst = o + ((size_t)t * p.num_kv_heads + hh) * dh;
    }
    if (dst == nullptr) continue;  // uniform over the warp

    if (kind == 2) {
      for (int i = lane; i < dv; i += 32) dst[i] = from_f32<T>(to_f32(src[i]));
      continue;
    }
    const float* w = kind == 0 ? p.q_norm_w : p.k_norm_w;
    float ss = 0.f;
    for (int i = lane; i < d; i += 32) {
      const float x = to_f32(src[i]);
      buf[i] = x;
      ss += x * x;
    }
    __syncwarp();
    if (w) {
      ss = warp_sum(ss);
      const float inv = rsqrtf(ss / (float)d + p.eps);
      // No rounding between norm and rotation: one rounding at the store.
      for (int i = lane; i < d; i += 32) buf[i] = buf[i] * inv * w[i];
      __syncwarp();
    }
    if (p.pairs || p.unit || p.temp_every > 0) {
      // rotated in place in shared memory, then divided, then stored
      if (p.inv_freq) {
        for (int i = lane; i < half; i += 32) {
          float s, c;
          sincosf((float)pos * p.inv_freq[i], &s, &c);
          s *= p.rot_scale; c *= p.rot_scale;
          const int a = p.pairs ? 2 * i : i, b = p.pairs ? 2 * i + 1 : i + half;
          const float x = buf[a], y = buf[b];
          buf[a] = x * c - y * s;
          buf[b] = x * s + y * c;
        }
        __syncwarp();
      }
      float f = 1.f;
      if (p.unit) {
        float s2 = 0.f;
        for (int i = lane; i < d; i += 32) s2 += buf[i] * buf[i];
        f = rsqrtf(warp_sum(s2) / (float)d + p.eps);
      }
      if (kind == 0) f *= temp;
      for (int i = lane; i < d; i += 32) dst[i] = from_f32<T>(buf[i] * f);
    } else if (p.inv_freq) {
      for (int i = lane; i < half; i += 32) {
        const float angle = (float)pos * p.inv_freq[i];
        float s, c;
        sincosf(angle, &s, &c);
        s *= p.rot_scale; c *= p.rot_scale;
        const float x = buf[i], y = buf[i + half];
        dst[i] = from_f32<T>(x * c - y * s);
        dst[i + half] = from_f32<T>(x * s + y * c);
      }
      for (int i = p.rot_dim + lane; i < d; i += 32) dst[i] = from_f32<T>(buf[i]);
    } else {
      for (int i = lane; i < d; i += 32) dst[i] = from_f32<T>(buf[i]);
    }
    __syncwarp();
  }
}

// The same for bfloat16 heads of 64, 128 or 256 elements with the whole head rotated: a lane holds
// VEC = d / 32 consecutive elements in registers (one 4-, 8- or 16-byte access), lanes 0..15 the first
// half of the head and lanes 16..31 the second, so the partner of a pair is the lane 16 further on.
template <int VEC>
__global__ void rope_kv_vec_kernel(RopeKvParams p) {
  pdl_trigger();
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  constexpr int d = VEC * 32;
  const int pos = p.positions[t];
  const int total_heads = p.num_q_heads + 2 * p.num_kv_heads;
  typedef typename std::conditional<VEC == 2, uint32_t, typename std::conditional<VEC == 4, uint2, uint4>::type>::type Word;
  // The angles depend on the token and the lane only: one sine and cosine per element for all heads
  // this warp walks over.
  float cs[VEC], sn[VEC];
  if (p.inv_freq) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      sincosf((float)pos * p.inv_freq[(lane & 15) * VEC + i], &sn[i], &cs[i]);
      sn[i] *= p.rot_scale; cs[i] *= p.rot_scale;
    }
  }
  // The token's page does not depend on the kernel ahead either (positions and block tables are the step's inputs).
  int page = -1;
  if (p.k_cache) page = p.block_table[(size_t)p.token_seq[t] * p.max_pages + pos / p.page_size];
  pdl_wait();                                   // what follows reads the q|k|v product
  // Four heads at a time: their loads are issued together, so that a warp keeps a kilobyte in flight
  // instead of 256 bytes.
  constexpr int UNR = 4;
  const int hstep = gridDim.y * nwarps;
  for (int h0 = blockIdx.y * nwarps + warp; h0 < total_heads; h0 += UNR * hstep) {
    Word raw[UNR];
    bf16* dsts[UNR];
    int kinds[UNR];
#pragma unroll
    for (int u = 0; u < UNR; ++u) {
      const int h = h0 + u * hstep;
      dsts[u] = nullptr; kinds[u] = 2;
      if (h >= total_heads) continue;
      const int kind = h < p.num_q_heads ? 0 : (h < p.num_q_heads + p.num_kv_heads ? 1 : 2);
      const int hh = kind == 0 ? h : (kind == 1 ? h - p.num_q_heads : h - p.num_q_heads - p.num_kv_heads);
      const bf16* src = kind == 0 ? (const bf16*)p.q_in + (size_t)t * p.q_stride + (size_t)hh * d
                      : kind == 1 ? (const bf16*)p.k_in + (size_t)t * p.k_stride + (size_t)hh * d
                                  : (const bf16*)p.v_in + (size_t)t * p.v_stride + (size_t)hh * d;
      bf16* dst = nullptr;
      if (kind == 0) {
        dst = (bf16*)p.q_out + ((size_t)t * p.num_q_heads + hh) * d;
      } else if (p.k_cache) {
        if (page >= 0) {
          bf16* pool = (bf16*)(kind == 1 ? p.k_cache : p.v_cache);
          dst = pool + (((size_t)page * p.num_kv_heads + hh) * p.page_size + pos % p.page_size) * d;
        }
      } else {
        bf16* o = (bf16*)(kind == 1 ? p.k_out : p.v_out);
        if (o) dst = o + ((size_t)t * p.num_kv_heads + hh) * d;
      }
      dsts[u] = dst; kinds[u] = kind;
      if (dst) raw[u] = reinterpret_cast<const Word*>(src)[lane];
    }
#pragma unroll
    for (int u = 0; u < UNR; ++u) {
      bf16* dst = dsts[u];
      if (dst == nullptr) continue;
      const int kind = kinds[u];
      if (kind == 2) { reinterpret_cast<Word*>(dst)[lane] = raw[u]; continue; }
      const bf16* e = reinterpret_cast<const bf16*>(&raw[u]);
      float x[VEC];
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < VEC; ++i) { x[i] = __bfloat162float(e[i]); ss += x[i] * x[i]; }
      const float* w = kind == 0 ? p.q_norm_w : p.k_norm_w;
      if (w) {
        ss = warp_sum(ss);
        const float inv = rsqrtf(ss / (float)d + p.eps);
#pragma unroll
        for (int i = 0; i < VEC; ++i) x[i] = x[i] * inv * w[lane * VEC + i];
      }
      if (p.inv_freq) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          const float other = __shfl_xor_sync(0xffffffffu, x[i], 16);
          // first half: x cos - y sin with y the partner; second half: x' sin + y' cos with x' the partner
          x[i] = lane < 16 ? x[i] * cs[i] - other * sn[i] : other * sn[i] + x[i] * cs[i];
        }
      }
      Word outw;
      bf16* o = reinterpret_cast<bf16*>(&outw);
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[i] = __float2bfloat16_rn(x[i]);
      reinterpret_cast<Word*>(dst)[lane] = outw;
    }
  }
}

// Neighbours as pairs, heads of up to 256 entries whose sizes are multiples of 4: a lane holds four consecutive entries
// of a head, two whole pairs, NV times (128 entries apart), so the rotation never leaves the lane; its sines and cosines
// are formed once for all heads the warp walks over (1 and 0 behind the rotated part).  q and k heads may be normed with
// a weight before the rotation, or divided by their root mean square behind it (`unit`).
__device__ __forceinline__ float4 rp_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 rp_load4(const bf16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
  return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void rp_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void rp_store4(bf16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}

template <typename T, typename TI, int NV>
__global__ void rope_pairs_kernel(RopeKvParams p) {
  pdl_trigger();
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  const int d = p.head_dim, dv = p.v_dim;
  const int pos = p.positions[t];
  const float temp = query_temperature(p, pos);
  const int total_heads = p.num_q_heads + 2 * p.num_kv_heads;
  float2 cs[NV], sn[NV];
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    float c[2], s[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int pair = n * 64 + lane * 2 + e;
      c[e] = 1.f; s[e] = 0.f;
      if (p.inv_freq && 2 * pair < p.rot_dim) {
        sincosf((float)pos * p.inv_freq[pair], &s[e], &c[e]);
        s[e] *= p.rot_scale; c[e] *= p.rot_scale;
      }
    }
    cs[n] = make_float2(c[0], c[1]); sn[n] = make_float2(s[0], s[1]);
  }
  int page = -1;
  if (p.k_cache) page = p.block_table[(size_t)p.token_seq[t] * p.max_pages + pos / p.page_size];
  pdl_wait();                                   // what follows reads the q|k|v product
  constexpr int UNR = NV == 1 ? 4 : 2;          // heads whose loads are issued together
  const int hstep = gridDim.y * nwarps;
  for (int h0 = blockIdx.y * nwarps + warp; h0 < total_heads; h0 += UNR * hstep) {
    float4 x[UNR][NV];
    T* dsts[UNR];
    int kinds[UNR];
#pragma unroll
    for (int u = 0; u < UNR; ++u) {
      const int h = h0 + u * hstep;
      dsts[u] = nullptr; kinds[u] = 2;
      if (h >= total_heads) continue;
      const int kind = h < p.num_q_heads ? 0 : (h < p.num_q_heads + p.num_kv_heads ? 1 : 2);
      const int hh = kind == 0 ? h : (kind == 1 ? h - p.num_q_heads : h - p.num_q_heads - p.num_kv_heads);
      const int dh = kind == 2 ? dv : d;
      const TI* src = kind == 0 ? (const TI*)p.q_in + (size_t)t * p.q_stride + (size_t)hh * d
                    : kind == 1 ? (const TI*)p.k_in + (size_t)t * p.k_stride + (size_t)hh * d
                                : (const TI*)p.v_in + (size_t)t * p.v_stride + (size_t)hh * dv;
      T* dst = nullptr;
      if (kind == 0) {
        dst = (T*)p.q_out + ((size_t)t * p.num_q_heads + hh) * d;
      } else if (p.k_cache) {
        if (page >= 0)
          dst = (T*)(kind == 1 ? p.k_cache : p.v_cache) + (((size_t)page * p.num_kv_heads + hh) * p.page_size + pos % p.page_size) * dh;
      } else {
        T* o = (T*)(kind == 1 ? p.k_out : p.v_out);
        if (o) dst = o + ((size_t)t * p.num_kv_heads + hh) * dh;
      }
      dsts[u] = dst; kinds[u] = kind;
      if (dst) {
#pragma unroll
        for (int n = 0; n < NV; ++n) {
          const int c = n * 128 + lane * 4;
          x[u][n] = c < dh ? rp_load4(src + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
      }
    }
#pragma unroll
    for (int u = 0; u < UNR; ++u) {
      T* dst = dsts[u];
      if (dst == nullptr) continue;             // uniform over the warp
      const int kind = kinds[u];
      if (kind != 2) {
        const float* w = kind == 0 ? p.q_norm_w : p.k_norm_w;
        if (w) {
          float ss = 0.f;
#pragma unroll
          for (int n = 0; n < NV; ++n) ss += x[u][n].x * x[u][n].x + x[u][n].y * x[u][n].y + x[u][n].z * x[u][n].z + x[u][n].w * x[u][n].w;
          const float f = rsqrtf(warp_sum(ss) / (float)d + p.eps);
#pragma unroll
          for (int n = 0; n < NV; ++n) {
            const int c = n * 128 + lane * 4;
            if (c < d) { x[u][n].x *= f * w[c]; x[u][n].y *= f * w[c + 1]; x[u][n].z *= f * w[c + 2]; x[u][n].w *= f * w[c + 3]; }
          }
        }
        float ss = 0.f;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
          const float4 a = x[u][n];
          x[u][n] = make_float4(a.x * cs[n].x - a.y * sn[n].x, a.x * sn[n].x + a.y * cs[n].x,
                                a.z * cs[n].y - a.w * sn[n].y, a.z * sn[n].y + a.w * cs[n].y);
          ss += x[u][n].x * x[u][n].x + x[u][n].y * x[u][n].y + x[u][n].z * x[u][n].z + x[u][n].w * x[u][n].w;
        }
        if (p.unit || (kind == 0 && p.temp_every > 0)) {
          const float f = (p.unit ? rsqrtf(warp_sum(ss) / (float)d + p.eps) : 1.f) * (kind == 0 ? temp : 1.f);
#pragma unroll
          for (int n = 0; n < NV; ++n) { x[u][n].x *= f; x[u][n].y *= f; x[u][n].z *= f; x[u][n].w *= f; }
        }
      }
      const int dh = kind == 2 ? dv : d;
#pragma unroll
      for (int n = 0; n < NV; ++n) {
        const int c = n * 128 + lane * 4;
        if (c < dh) rp_store4(dst + c, x[u][n]);
      }
    }
  }
}

// Rotation in place of 32-bit rows, for mixers that keep q and k in 32-bit (no cache, no norm): up to two column
// ranges of x [T, ld], each `heads` heads of `head_dim`, whose first rot_dim entries are rotated as above and whose
// every entry is then multiplied by the range's `scale`.  One warp a head.
struct RotateRowsParams {
  float* x; long long ld;
  const int* positions; const float* inv_freq;
  int head_dim, rot_dim;
  float rot_scale;
  int col[2], heads[2];
  float scale[2];
};

__global__ void rotate_rows_kernel(RotateRowsParams p) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  const int half = p.rot_dim >> 1, d = p.head_dim;
  const int pos = p.positions[t];
  const int total = p.heads[0] + p.heads[1];
  for (int h = blockIdx.y * nwarps + warp; h < total; h += gridDim.y * nwarps) {
    const int r = h < p.heads[0] ? 0 : 1;
    float* row = p.x + (size_t)t * p.ld + p.col[r] + (size_t)(r == 0 ? h : h - p.heads[0]) * d;
    const float sc = p.scale[r];
    for (int i = lane; i < half; i += 32) {
      float s, c;
      sincosf((float)pos * p.inv_freq[i], &s, &c);
      s *= p.rot_scale; c *= p.rot_scale;
      const float x = row[i], y = row[i + half];
      row[i] = (x * c - y * s) * sc;
      row[i + half] = (x * s + y * c) * sc;
    }
    if (sc != 1.f)
      for (int i = p.rot_dim + lane; i < d; i += 32) row[i] *= sc;
  }
}

}  // namespace lb

LB_EXPORT int lb_rotate_rows(float* x, long long ld, int num_tokens, const int* positions, const float* inv_freq, int head_dim,
                             int rot_dim, float rot_scale, int col0, int heads0, float scale0, int col1, int heads1, float scale1,
                             cudaStream_t stream) {
  LB_CHECK_ARG(x && positions && head_dim > 0 && rot_dim >= 0 && rot_dim <= head_dim && rot_dim % 2 == 0 && (rot_dim == 0 || inv_freq),
               "rotate_rows: rotary size %d must be even and at most head_dim %d", rot_dim, head_dim);
  LB_CHECK_ARG(heads0 >= 0 && heads1 >= 0 && col0 >= 0 && col1 >= 0 && num_tokens >= 0, "rotate_rows: bad ranges");
  if (num_tokens == 0 || heads0 + heads1 == 0) return 0;
  lb::RotateRowsParams p;
  p.x = x; p.ld = ld; p.positions = positions; p.inv_freq = inv_freq; p.head_dim = head_dim; p.rot_dim = rot_dim;
  p.rot_scale = rot_scale; p.col[0] = col0; p.col[1] = col1; p.heads[0] = heads0; p.heads[1] = heads1;
  p.scale[0] = scale0; p.scale[1] = scale1;
  const int warps = 4;
  int head_blocks = (heads0 + heads1 + warps - 1) / warps;
  if (head_blocks > 64) head_blocks = 64;
  lb::launch(lb::rotate_rows_kernel, dim3(num_tokens, head_blocks), dim3(warps * 32), 0, stream, p);
  LB_CHECK_LAUNCH("rotate_rows");
  return 0;
}

LB_EXPORT int lb_rope_kv(int dtype, const void* q_in, const void* k_in, const void* v_in,
                         long long q_stride, long long k_stride, long long v_stride, void* q_out,
                         void* k_out, void* v_out, void* k_cache, void* v_cache,
                         const int* positions, const int* token_seq, const int* block_table,
                         const float* q_norm_w, const float* k_norm_w, const float* inv_freq,
                         int num_tokens, int num_q_heads, int num_kv_heads, int head_dim,
                         int rot_dim, int page_size, int max_pages, float eps, int in_dtype, int v_dim,
                         float rot_scale, int pairs, int unit, float temp_coef, int temp_every, cudaStream_t stream) {
  if (v_dim <= 0) v_dim = head_dim;
  LB_CHECK_ARG(lb::valid_dtype(in_dtype) && v_dim <= 1024, "rope_kv: bad input type or value size");
  LB_CHECK_ARG(lb::valid_dtype(dtype), "rope_kv: bad dtype %d", dtype);
  LB_CHECK_ARG(head_dim > 0 && head_dim <= 1024, "rope_kv: head_dim %d not in 1..1024", head_dim);
  LB_CHECK_ARG(rot_dim >= 0 && rot_dim <= head_dim && rot_dim % 2 == 0,
               "rope_kv: rotary size %d must be even and at most head_dim %d", rot_dim, head_dim);
  LB_CHECK_ARG(num_q_heads >= 0 && num_kv_heads >= 0, "rope_kv: bad head counts");
  LB_CHECK_ARG(k_cache == nullptr || (v_cache && block_table && token_seq && page_size > 0 && max_pages > 0),
               "rope_kv: a cache needs v pool, block table, token map and page size");
  if (num_tokens == 0) return 0;
  lb::RopeKvParams p;
  p.q_in = q_in; p.k_in = k_in; p.v_in = v_in;
  p.q_stride = q_stride; p.k_stride = k_stride; p.v_stride = v_stride;
  p.q_out = q_out; p.k_out = k_out; p.v_out = v_out; p.k_cache = k_cache; p.v_cache = v_cache;
  p.positions = positions; p.token_seq = token_seq; p.block_table = block_table;
  p.q_norm_w = q_norm_w; p.k_norm_w = k_norm_w; p.inv_freq = rot_dim > 0 ? inv_freq : nullptr;
  p.num_q_heads = num_q_heads; p.num_kv_heads = num_kv_heads; p.head_dim = head_dim;
  p.rot_dim = rot_dim; p.page_size = page_size; p.max_pages = max_pages; p.eps = eps; p.v_dim = v_dim;
  p.rot_scale = rot_scale; p.pairs = pairs; p.unit = unit; p.temp_coef = temp_coef; p.temp_every = temp_every;
  LB_CHECK_ARG(temp_every >= 0, "rope_kv: a temperature that grows every %d positions", temp_every);
  LB_CHECK_ARG(!unit || (q_norm_w == nullptr && k_norm_w == nullptr), "rope_kv: heads are normed in front of the rotation or behind it, not both");
  const int warps = 4;
  // (without a rotation how entries pair does not matter: that kernel then serves unit heads of either kind)
  if ((pairs || (unit && p.inv_freq == nullptr)) && head_dim % 4 == 0 && v_dim % 4 == 0 && head_dim <= 256 && v_dim <= 256) {
    const int in_el = in_dtype == LB_F32 ? 4 : 2, el = dtype == LB_F32 ? 4 : 2;
    auto in_ok = [&](const void* ptr, long long stride) { return (uintptr_t)ptr % (4 * in_el) == 0 && stride % 4 == 0; };
    auto out_ok = [&](const void* ptr) { return (uintptr_t)ptr % (4 * el) == 0; };
    if (in_ok(q_in, q_stride) && in_ok(k_in, k_stride) && in_ok(v_in, v_stride) && out_ok(q_out) && out_ok(k_out) && out_ok(v_out) && out_ok(k_cache) &&
        out_ok(v_cache)) {
      const int total_heads = num_q_heads + 2 * num_kv_heads;
      int head_blocks = (total_heads + warps - 1) / warps;
      const int wanted = (1184 + num_tokens - 1) / num_tokens;      // near eight blocks per SM, as below
      if (head_blocks > wanted) head_blocks = wanted;
      if (head_blocks < 1) head_blocks = 1;
      const bool two = head_dim > 128 || v_dim > 128;
      LB_DISPATCH_DTYPE(dtype, T, {
        LB_DISPATCH_DTYPE(in_dtype, TI, {
          if (two) lb::launch(lb::rope_pairs_kernel<T, TI, 2>, dim3(num_tokens, head_blocks), dim3(warps * 32), 0, stream, p);
          else lb::launch(lb::rope_pairs_kernel<T, TI, 1>, dim3(num_tokens, head_blocks), dim3(warps * 32), 0, stream, p);
        })
      })
      LB_CHECK_LAUNCH("rope_kv");
      return 0;
    }
  }
  const size_t smem = (size_t)warps * head_dim * sizeof(float);
  // The register version: bfloat16, heads of 64 / 128 / 256, whole head rotated, every row 16-byte aligned.
  const int vec = head_dim / 32;
  const size_t word = (size_t)vec * 2;
  auto aligned = [&](const void* ptr, long long stride) { return ptr == nullptr || ((uintptr_t)ptr % word == 0 && (stride * 2) % (long long)word == 0); };
  const bool fast = !pairs && !unit && temp_every == 0 && dtype == LB_BF16 && in_dtype == LB_BF16 && v_dim == head_dim && (head_dim == 64 || head_dim == 128 || head_dim == 256) &&
                    (p.inv_freq == nullptr || rot_dim == head_dim) && aligned(q_in, q_stride) && aligned(k_in, k_stride) &&
                    aligned(v_in, v_stride) && aligned(q_out, head_dim) && aligned(k_out, head_dim) && aligned(v_out, head_dim) &&
                    aligned(k_cache, head_dim) && aligned(v_cache, head_dim);
  if (fast) {
    // With few tokens every head gets a warp of its own; with many a warp walks over several heads,
    // so that the grid stays near eight blocks per SM instead of tens of thousands of tiny ones.
    const int total_heads = num_q_heads + 2 * num_kv_heads;
    int head_blocks = (total_heads + warps - 1) / warps;
    const int wanted = (1184 + num_tokens - 1) / num_tokens;
    if (head_blocks > wanted) head_blocks = wanted;
    if (head_blocks < 1) head_blocks = 1;
    dim3 grid(num_tokens, head_blocks);
    if (vec == 2) lb::launch(lb::rope_kv_vec_kernel<2>, grid, dim3(warps * 32), 0, stream, p);
    else if (vec == 4) lb::launch(lb::rope_kv_vec_kernel<4>, grid, dim3(warps * 32), 0, stream, p);
    else lb::launch(lb::rope_kv_vec_kernel<8>, grid, dim3(warps * 32), 0, stream, p);
    LB_CHECK_LAUNCH("rope_kv");
    return 0;
  }
  LB_DISPATCH_DTYPE(dtype, T, {
    const int total_heads = num_q_heads + 2 * num_kv_heads;
    int head_blocks = (total_heads + warps - 1) / warps;
    if (head_blocks > 65535) head_blocks = 65535;
    if (head_blocks < 1) head_blocks = 1;
    LB_DISPATCH_DTYPE(in_dtype, TI, {
      lb::launch(lb::rope_kv_kernel<T, TI>, dim3(num_tokens, head_blocks), dim3(warps * 32), smem, stream, p);
    })
  })
  LB_CHECK_LAUNCH("rope_kv");
  return 0;
}
