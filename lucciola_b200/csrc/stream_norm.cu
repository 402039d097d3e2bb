// What stands between two products of a model that norms a sublayer's OUTPUT before it adds it to the residual stream
// and norms the stream again in front of the next sublayer, as one pass over the row:
//
//   y        = y_in                                     a sublayer's output (32-bit or bfloat16), or, from routed experts,
//              sum_k weight * e[place(t, k)] [+ sigmoid(g . x_t) * s_t]      their weighted sum formed here (below)
//   v        = residual + add0 + add1 + vec + y / sqrt(mean(y^2) + y_eps) * y_w       every term but the first optional
//   residual = v                                         (not when a row list is given, nor when `lo` is)
//   out      = v / sqrt(mean(v^2) + eps) * w             (with w)
//   or, without w:  out = v rounded to bfloat16, lo = v - out rounded again: the row in two parts that carry 16 of its bits,
//              for a product whose operands are bfloat16 and whose input is the stream itself
//
// vec is one vector for all rows.  Everything is 32-bit, each row is one CTA's, and the order of every sum is fixed by
// the row's length, never by the batch.
//
// Experts: a token's chosen experts' rows e[place] (32-bit) are added in the order of the choice, each times one
// constant weight or its own; the expert every token uses (s, 32-bit or bfloat16) is added times the sigmoid of one
// number a token, formed here from the sublayer's input x (the row the products read) and the weights g.
#include "common.cuh"

namespace lb {

struct StreamNormParams {
  void* out; void* lo;                 // lo: the second part (bfloat16), with w == nullptr only
  float* residual;
  const float* add0; const float* add1; const float* vec;
  const void* y; const float* y_w; float y_eps;
  const float* w; float eps;
  const int* rows;
  int hidden;
  // experts (y == nullptr, e != nullptr)
  const float* e; const int* place_of; const float* weights; int top; float weight;
  const void* shared; const void* x; const float* gate;
};

__device__ __forceinline__ float4 sn_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 sn_load4(const bf16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
  return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void sn_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void sn_store4(bf16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}
__device__ __forceinline__ float4 sn_add(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float4 sn_fma(float s, float4 a, float4 c) {
  return make_float4(fmaf(s, a.x, c.x), fmaf(s, a.y, c.y), fmaf(s, a.z, c.z), fmaf(s, a.w, c.w));
}
__device__ __forceinline__ float sn_sq(float4 a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }

// Rows that fit the CTA's registers: a thread holds PER vectors of four elements, those at 4 * (q * threads + thread);
// the last ones may lie past the row's end.  TY: the sublayer's output (and the shared expert's), TX: the sublayer's input.
template <typename TY, typename TO, typename TX, int PER, bool EXPERTS>
__global__ void __launch_bounds__(PER == 1 ? 128 : 1024) stream_norm_row_kernel(StreamNormParams p) {
  __shared__ float scratch[33];
  pdl_trigger();
  const int tid = threadIdx.x, nt = blockDim.x, n4 = p.hidden >> 2;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 yw[PER], w[PER], v[PER], y[PER];
  bool in[PER];
  int at[PER];
#pragma unroll
  for (int q = 0; q < PER; ++q) { at[q] = 4 * (q * nt + tid); in[q] = q * nt + tid < n4; }
  const bool normed = p.y != nullptr || EXPERTS;
#pragma unroll
  for (int q = 0; q < PER; ++q) {             // what no kernel of the step writes is read before the wait
    yw[q] = normed && in[q] ? sn_load4(p.y_w + at[q]) : zero;
    w[q] = p.w && in[q] ? sn_load4(p.w + at[q]) : zero;
  }
  pdl_wait();
  const int i = blockIdx.x;
  const size_t src = (size_t)(p.rows ? p.rows[i] : i);
  float* r = p.residual + src * p.hidden;
#pragma unroll
  for (int q = 0; q < PER; ++q) v[q] = in[q] ? sn_load4(r + at[q]) : zero;
  if (EXPERTS) {
    float g = 0.f;
    if (p.gate) {
      const TX* x = (const TX*)p.x + src * p.hidden;
      float part = 0.f;
#pragma unroll
      for (int q = 0; q < PER; ++q)
        if (in[q]) {
          const float4 a = sn_load4(x + at[q]), b = sn_load4(p.gate + at[q]);
          part += a.x * b.x + a.y * b.y + a.z * b.z + a.w * b.w;
        }
      g = 1.f / (1.f + expf(-block_sum(part, scratch)));
    }
#pragma unroll
    for (int q = 0; q < PER; ++q) y[q] = zero;
    for (int k0 = 0; k0 < p.top; k0 += 2) {     // two choices' rows in flight at a time, added in order
      float wk[2];
      const float* e[2];
      float4 t[2][PER];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const bool have = k0 + u < p.top;
        const size_t pair = src * p.top + k0 + (have ? u : 0);
        e[u] = p.e + (size_t)p.place_of[pair] * p.hidden;
        wk[u] = have ? (p.weights ? p.weights[pair] : p.weight) : 0.f;
      }
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int q = 0; q < PER; ++q) t[u][q] = in[q] && k0 + u < p.top ? sn_load4(e[u] + at[q]) : zero;
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int q = 0; q < PER; ++q) y[q] = sn_fma(wk[u], t[u][q], y[q]);
    }
    if (p.shared) {
      const TY* s = (const TY*)p.shared + src * p.hidden;
      const float gs = p.gate ? g : 1.f;
#pragma unroll
      for (int q = 0; q < PER; ++q)
        if (in[q]) y[q] = sn_fma(gs, sn_load4(s + at[q]), y[q]);
    }
  } else if (p.y) {
    const TY* yr = (const TY*)p.y + src * p.hidden;
#pragma unroll
    for (int q = 0; q < PER; ++q) y[q] = in[q] ? sn_load4(yr + at[q]) : zero;
  }
  if (p.add0) {
    const float* a = p.add0 + src * p.hidden;
#pragma unroll
    for (int q = 0; q < PER; ++q) if (in[q]) v[q] = sn_add(v[q], sn_load4(a + at[q]));
  }
  if (p.add1) {
    const float* a = p.add1 + src * p.hidden;
#pragma unroll
    for (int q = 0; q < PER; ++q) if (in[q]) v[q] = sn_add(v[q], sn_load4(a + at[q]));
  }
  if (p.vec) {
#pragma unroll
    for (int q = 0; q < PER; ++q) if (in[q]) v[q] = sn_add(v[q], sn_load4(p.vec + at[q]));
  }
  if (normed) {
    float ss = 0.f;
#pragma unroll
    for (int q = 0; q < PER; ++q) ss += sn_sq(y[q]);
    const float f = rsqrtf(block_sum(ss, scratch) / (float)p.hidden + p.y_eps);
#pragma unroll
    for (int q = 0; q < PER; ++q)
      v[q] = make_float4(v[q].x + y[q].x * f * yw[q].x, v[q].y + y[q].y * f * yw[q].y, v[q].z + y[q].z * f * yw[q].z, v[q].w + y[q].w * f * yw[q].w);
  }
  const bool update = p.rows == nullptr && p.lo == nullptr && (normed || p.add0 || p.add1 || p.vec);
  if (update) {
#pragma unroll
    for (int q = 0; q < PER; ++q) if (in[q]) sn_store4(r + at[q], v[q]);
  }
  if (p.w) {
    float ss = 0.f;
#pragma unroll
    for (int q = 0; q < PER; ++q) ss += sn_sq(v[q]);
    const float f = rsqrtf(block_sum(ss, scratch) / (float)p.hidden + p.eps);
    TO* o = (TO*)p.out + (size_t)i * p.hidden;
#pragma unroll
    for (int q = 0; q < PER; ++q)
      if (in[q]) sn_store4(o + at[q], make_float4(v[q].x * f * w[q].x, v[q].y * f * w[q].y, v[q].z * f * w[q].z, v[q].w * f * w[q].w));
  } else if (p.lo) {
    bf16* hi = (bf16*)p.out + (size_t)i * p.hidden;
    bf16* lo = (bf16*)p.lo + (size_t)i * p.hidden;
#pragma unroll
    for (int q = 0; q < PER; ++q)
      if (in[q]) {
        const float4 h = make_float4(__bfloat162float(__float2bfloat16_rn(v[q].x)), __bfloat162float(__float2bfloat16_rn(v[q].y)),
                                     __bfloat162float(__float2bfloat16_rn(v[q].z)), __bfloat162float(__float2bfloat16_rn(v[q].w)));
        sn_store4(hi + at[q], h);
        sn_store4(lo + at[q], make_float4(v[q].x - h.x, v[q].y - h.y, v[q].z - h.z, v[q].w - h.w));
      }
  }
}

// Any row length: an element at a time, the row formed again in every pass.
template <typename TY, typename TO, typename TX>
__global__ void stream_norm_any_kernel(StreamNormParams p) {
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x;
  const size_t src = (size_t)(p.rows ? p.rows[i] : i);
  const size_t base = src * p.hidden;
  float* r = p.residual + base;
  const bool normed = p.y != nullptr || p.e != nullptr;
  float g = 1.f;
  if (p.e && p.gate) {
    float part = 0.f;
    for (int j = threadIdx.x; j < p.hidden; j += blockDim.x) part += to_f32(((const TX*)p.x)[base + j]) * p.gate[j];
    g = 1.f / (1.f + expf(-block_sum(part, scratch)));
  }
  auto y_of = [&](int j) -> float {
    if (p.y) return to_f32(((const TY*)p.y)[base + j]);
    float acc = 0.f;
    for (int k = 0; k < p.top; ++k) {
      const size_t pair = src * p.top + k;
      acc = fmaf(p.weights ? p.weights[pair] : p.weight, p.e[(size_t)p.place_of[pair] * p.hidden + j], acc);
    }
    if (p.shared) acc = fmaf(g, to_f32(((const TY*)p.shared)[base + j]), acc);
    return acc;
  };
  float fy = 0.f;
  if (normed) {
    float ss = 0.f;
    for (int j = threadIdx.x; j < p.hidden; j += blockDim.x) { const float y = y_of(j); ss += y * y; }
    fy = rsqrtf(block_sum(ss, scratch) / (float)p.hidden + p.y_eps);
  }
  auto v_of = [&](int j) -> float {
    float v = r[j];
    if (p.add0) v += p.add0[base + j];
    if (p.add1) v += p.add1[base + j];
    if (p.vec) v += p.vec[j];
    if (normed) v += y_of(j) * fy * p.y_w[j];
    return v;
  };
  const bool changes = normed || p.add0 || p.add1 || p.vec;
  const bool update = p.rows == nullptr && p.lo == nullptr && changes;
  if (p.w) {
    float ss = 0.f;
    for (int j = threadIdx.x; j < p.hidden; j += blockDim.x) {
      const float v = v_of(j);
      if (update) r[j] = v;                      // this thread's element: read again below as written here
      ss += v * v;
    }
    const float f = rsqrtf(block_sum(ss, scratch) / (float)p.hidden + p.eps);
    TO* o = (TO*)p.out + (size_t)i * p.hidden;
    for (int j = threadIdx.x; j < p.hidden; j += blockDim.x) o[j] = from_f32<TO>((update ? r[j] : v_of(j)) * f * p.w[j]);
    return;
  }
  for (int j = threadIdx.x; j < p.hidden; j += blockDim.x) {
    const float v = v_of(j);
    if (update) r[j] = v;
    if (p.lo) {
      const bf16 h = __float2bfloat16_rn(v);
      ((bf16*)p.out)[(size_t)i * p.hidden + j] = h;
      ((bf16*)p.lo)[(size_t)i * p.hidden + j] = __float2bfloat16_rn(v - __bfloat162float(h));
    }
  }
}

template <typename TY, typename TO, typename TX>
void launch_stream_norm(const StreamNormParams& p, int num_rows, bool vec, cudaStream_t stream) {
  const int n4 = p.hidden >> 2;
  // vectors of four elements a thread: one for short rows, else two; a whole number of warps, at most 1024 threads
  const int per = n4 <= 128 ? 1 : 2;
  const int threads = ((n4 + per - 1) / per + 31) / 32 * 32;
  if (vec && threads <= 1024) {
#define LB_SN(PER, EX) launch(stream_norm_row_kernel<TY, TO, TX, PER, EX>, dim3(num_rows), dim3(threads), 0, stream, p)
    if (p.e) { if (per == 1) LB_SN(1, true); else LB_SN(2, true); }
    else { if (per == 1) LB_SN(1, false); else LB_SN(2, false); }
#undef LB_SN
  } else {
    const int t = p.hidden >= 2048 ? 512 : (p.hidden >= 512 ? 256 : 64);
    launch(stream_norm_any_kernel<TY, TO, TX>, dim3(num_rows), dim3(t), 0, stream, p);
  }
}

}  // namespace lb

// One row for each of num_rows (rows[i] of the operands if `rows` is given).  y_dtype: type of y, or of `shared`; x_dtype: of
// x.  Either y, or the experts' e with place_of, or neither.  Without w: lo (bfloat16, with a bfloat16 out) asks for the
// two parts, neither for the update of the residual alone.
LB_EXPORT int lb_stream_norm(void* out, int out_dtype, void* lo, float* residual, const float* add0, const float* add1, const float* vec,
                             const void* y, int y_dtype, const float* y_w, float y_eps, const float* w, float eps, const int* rows,
                             const float* e, const int* place_of, const float* weights, int top, float weight, const void* shared,
                             const void* x, int x_dtype, const float* gate, int num_rows, int hidden, cudaStream_t stream) {
  LB_CHECK_ARG(lb::valid_dtype(out_dtype) && lb::valid_dtype(y_dtype) && lb::valid_dtype(x_dtype), "stream_norm: bad dtype");
  LB_CHECK_ARG(residual && num_rows >= 0 && hidden > 0, "stream_norm: bad sizes rows=%d hidden=%d", num_rows, hidden);
  LB_CHECK_ARG(!(y && e) && ((!y && !e) || y_w), "stream_norm: one output to be normed, with its norm's weight");
  LB_CHECK_ARG(!e || (place_of && top > 0), "stream_norm: experts' rows need the pairs' places");
  LB_CHECK_ARG((!shared || e) && (!gate || (shared && x)), "stream_norm: a gate goes with the shared expert's output and the sublayer's input");
  LB_CHECK_ARG(w ? (out != nullptr && lo == nullptr) : ((lo != nullptr) == (out != nullptr)), "stream_norm: a norm's output, two parts, or neither");
  LB_CHECK_ARG(!lo || out_dtype == LB_BF16, "stream_norm: the two parts are bfloat16");
  if (num_rows == 0) return 0;
  lb::StreamNormParams p;
  p.out = out; p.lo = lo; p.residual = residual; p.add0 = add0; p.add1 = add1; p.vec = vec; p.y = y; p.y_w = y_w; p.y_eps = y_eps;
  p.w = w; p.eps = eps; p.rows = rows; p.hidden = hidden; p.e = e; p.place_of = place_of; p.weights = weights; p.top = top;
  p.weight = weight; p.shared = shared; p.x = x; p.gate = gate;
  auto ok = [](const void* ptr) { return (uintptr_t)ptr % 16 == 0; };
  const bool vec4 = hidden % 4 == 0 && ok(out) && ok(lo) && ok(residual) && ok(add0) && ok(add1) && ok(vec) && ok(y) && ok(y_w) && ok(w) && ok(e) &&
                    ok(shared) && ok(x) && ok(gate);
  LB_DISPATCH_DTYPE(y_dtype, TY, {
    LB_DISPATCH_DTYPE(out_dtype, TO, {
      LB_DISPATCH_DTYPE(x_dtype, TX, { lb::launch_stream_norm<TY, TO, TX>(p, num_rows, vec4, stream); })
    })
  })
  LB_CHECK_LAUNCH("stream_norm");
  return 0;
}
