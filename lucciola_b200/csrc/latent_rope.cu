// Latent attention with a rotated part, the step between the product that reads the mixer's input and the attention: from the
// 32-bit sums of a token,
//
//   q    heads x [dim | rot], head by head at column q_col       -> q_out [T, heads, dim + rot], the last rot entries rotated,
//                                                                   and, if q_lat is given, the rotated part a second time
//                                                                   behind kv_rank places of q_lat [T, heads, kv_rank + rot]
//   c    kv_rank values at column kv_col, RMS-normed (weight)    -> the first kv_rank entries of the token's place in the pages
//   k    the rot values behind them, rotated                     -> the entries behind those
//
// Rotation: the first rot_dims of the rot entries, entries i and i + rot_dims/2 a pair turned by position * inv_freq[i], sines
// and cosines times rot_scale.  Everything is 32-bit up to the one rounding at each store; the angle is one 32-bit product.
// Page layout: [page][slot][kv_rank + rot] (one "head" whose values are the first kv_rank entries of its keys).
#include "common.cuh"

namespace lb {

struct LatentRopeParams {
  const float* pre; long long ld;
  int q_col, kv_col, heads, dim, rot, rot_dims, kv_rank;
  const float* kv_w; const float* inv_freq; float rot_scale;
  void* q_out; void* q_lat; void* pages;
  const int* positions; const int* token_seq; const int* block_table;
  int page_size, max_pages;
  float eps;
};

// four values to the activation type
__device__ __forceinline__ void lr_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void lr_store4(bf16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}

constexpr int LR_THREADS = 256, LR_HEADS_A_BLOCK = 16;

// block y = 0: the latent and the shared key part; blocks y >= 1: 16 heads of the query each, a warp a head.
// VEC: every column, size and pointer allows four values at a time.
template <typename T, bool VEC>
__global__ void __launch_bounds__(LR_THREADS) latent_rope_kernel(LatentRopeParams p) {
  extern __shared__ float cs[];                 // cosines, then sines, of the token's rot_dims / 2 angles
  __shared__ float scratch[33];
  pdl_trigger();
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int half = p.rot_dims >> 1;
  const int pos = p.positions[t];               // positions and block tables are the step's inputs
  for (int i = tid; i < half; i += LR_THREADS) {
    float s, c;
    sincosf((float)pos * p.inv_freq[i], &s, &c);
    cs[i] = c * p.rot_scale; cs[half + i] = s * p.rot_scale;
  }
  int page = -1;
  if (blockIdx.y == 0) page = p.block_table[(size_t)p.token_seq[t] * p.max_pages + pos / p.page_size];
  __syncthreads();
  pdl_wait();
  const float* row = p.pre + (size_t)t * p.ld;
  if (blockIdx.y == 0) {
    if (page < 0) return;                       // an entry that owns no page: uniform over the block
    const float* c = row + p.kv_col;
    T* dst = (T*)p.pages + ((size_t)page * p.page_size + pos % p.page_size) * (p.kv_rank + p.rot);
    float ss = 0.f;
    for (int i = tid; i < p.kv_rank; i += LR_THREADS) ss += c[i] * c[i];
    const float f = 1.f / sqrtf(block_sum(ss, scratch) / (float)p.kv_rank + p.eps);
    for (int i = tid; i < p.kv_rank; i += LR_THREADS) dst[i] = from_f32<T>(c[i] * f * p.kv_w[i]);
    const float* k = c + p.kv_rank;
    for (int i = tid; i < p.rot; i += LR_THREADS) {
      float v = k[i];
      if (i < half) v = k[i] * cs[i] - k[i + half] * cs[half + i];
      else if (i < 2 * half) v = k[i] * cs[i - half] + k[i - half] * cs[i];
      dst[p.kv_rank + i] = from_f32<T>(v);
    }
    return;
  }
  const int hd = p.dim + p.rot;
  const int h1 = min((int)blockIdx.y * LR_HEADS_A_BLOCK, p.heads);
  for (int h = ((int)blockIdx.y - 1) * LR_HEADS_A_BLOCK + warp; h < h1; h += LR_THREADS / 32) {
    const float* q = row + p.q_col + (size_t)h * hd;
    T* dst = (T*)p.q_out + ((size_t)t * p.heads + h) * hd;
    T* lat = p.q_lat ? (T*)p.q_lat + ((size_t)t * p.heads + h) * (p.kv_rank + p.rot) + p.kv_rank : nullptr;
    if (VEC) {
      for (int i = lane * 4; i < p.dim; i += 128) lr_store4(dst + i, *reinterpret_cast<const float4*>(q + i));
    } else {
      for (int i = lane; i < p.dim; i += 32) dst[i] = from_f32<T>(q[i]);
    }
    q += p.dim; dst += p.dim;
    for (int i = lane; i < half; i += 32) {
      const float u = q[i], v = q[i + half];
      const T a = from_f32<T>(u * cs[i] - v * cs[half + i]), b = from_f32<T>(v * cs[i] + u * cs[half + i]);
      dst[i] = a; dst[i + half] = b;
      if (lat) { lat[i] = a; lat[i + half] = b; }
    }
    for (int i = p.rot_dims + lane; i < p.rot; i += 32) {
      const T a = from_f32<T>(q[i]);
      dst[i] = a;
      if (lat) lat[i] = a;
    }
  }
}

}  // namespace lb

LB_EXPORT int lb_latent_rope(int dtype, const float* pre, long long ld, int q_col, int kv_col, int heads, int dim, int rot,
                             int rot_dims, int kv_rank, const float* kv_w, const float* inv_freq, float rot_scale, void* q_out,
                             void* q_lat, void* pages, const int* positions, const int* token_seq, const int* block_table,
                             int num_tokens, int page_size, int max_pages, float eps, cudaStream_t stream) {
  LB_CHECK_ARG(lb::valid_dtype(dtype), "latent_rope: bad dtype %d", dtype);
  LB_CHECK_ARG(num_tokens >= 0 && heads > 0 && dim >= 0 && rot >= 0 && dim + rot > 0 && kv_rank > 0 && page_size > 0 && max_pages > 0,
               "latent_rope: bad sizes");
  LB_CHECK_ARG(rot_dims >= 0 && rot_dims <= rot && rot_dims % 2 == 0 && rot_dims <= 4096 && (rot_dims == 0 || inv_freq),
               "latent_rope: rotary size %d must be even and at most %d", rot_dims, rot);
  LB_CHECK_ARG(pre && kv_w && q_out && pages && positions && token_seq && block_table, "latent_rope: null argument");
  if (num_tokens == 0) return 0;
  lb::LatentRopeParams p;
  p.pre = pre; p.ld = ld; p.q_col = q_col; p.kv_col = kv_col; p.heads = heads; p.dim = dim; p.rot = rot; p.rot_dims = rot_dims;
  p.kv_rank = kv_rank; p.kv_w = kv_w; p.inv_freq = inv_freq; p.rot_scale = rot_scale; p.q_out = q_out; p.q_lat = q_lat; p.pages = pages;
  p.positions = positions; p.token_seq = token_seq; p.block_table = block_table; p.page_size = page_size; p.max_pages = max_pages; p.eps = eps;
  const dim3 grid(num_tokens, 1 + (heads + lb::LR_HEADS_A_BLOCK - 1) / lb::LR_HEADS_A_BLOCK);
  const bool vec = dim % 4 == 0 && rot % 4 == 0 && q_col % 4 == 0 && ld % 4 == 0 && (uintptr_t)pre % 16 == 0 && (uintptr_t)q_out % 16 == 0;
  LB_DISPATCH_DTYPE(dtype, T, {
    if (vec) lb::launch(lb::latent_rope_kernel<T, true>, grid, dim3(lb::LR_THREADS), (size_t)rot_dims * sizeof(float), stream, p);
    else lb::launch(lb::latent_rope_kernel<T, false>, grid, dim3(lb::LR_THREADS), (size_t)rot_dims * sizeof(float), stream, p);
  })
  LB_CHECK_LAUNCH("latent_rope");
  return 0;
}
