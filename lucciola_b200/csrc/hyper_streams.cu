// What stands between two sublayers of a model that keeps S parallel residual streams, as one pass over a token's row:
//
//   y      = y_in                                   a sublayer's output (32-bit or bfloat16), or, from routed experts,
//            sum_k weight[t, k] * e[place(t, k)]     their weighted sum, formed here in the order of the choice
//   x_t    = sum_s mix[s, t] * x_s + out[t] * y      the streams behind that sublayer (without a mix they stay as they are)
//   u      = sum_t in[t] * x_t                       what the next sublayer reads (without `in`: the plain sum)
//   normed = u / sqrt(mean(u^2) + eps) * w
//
// Streams are 32-bit, [T, S, hidden].  At the start all S are one and the same row: then the input is [T, hidden] and
// every x_s means that row.  Behind the last sublayer only u is wanted, on the rows whose logits are computed: without
// x_new nothing of the streams is written.  Everything is 32-bit, a row is one CTA's, and the order of every sum is
// fixed by S and the row's length, never by the batch.
#include "common.cuh"

namespace lb {

struct StreamsParams {
  void* normed;
  const float* x; float* x_new;          // x_new may be x itself (a thread reads its columns of all streams before it writes them)
  int streams, same;                     // same: x is [T, hidden], one row for all streams
  const float* mix; const float* out; const float* in;      // [S, S] (from, to), [S], [S]
  const void* y;
  const float* e; const int* place_of; const float* weights; int top; float weight;
  const float* w; float eps;
  const int* rows;
  int hidden;
};

__device__ __forceinline__ float4 hs_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 hs_load4(const bf16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
  return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void hs_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void hs_store4(bf16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}
__device__ __forceinline__ float4 hs_fma(float s, float4 a, float4 c) {
  return make_float4(fmaf(s, a.x, c.x), fmaf(s, a.y, c.y), fmaf(s, a.z, c.z), fmaf(s, a.w, c.w));
}

// Rows that fit the CTA's registers: a thread holds PER vectors of four elements of every stream, those at
// 4 * (q * threads + thread).  S: the number of streams.
template <typename TY, typename TO, int S, int PER>
__global__ void __launch_bounds__(1024) streams_row_kernel(StreamsParams p) {
  __shared__ float scratch[33];
  pdl_trigger();
  const int tid = threadIdx.x, nt = blockDim.x, n4 = p.hidden >> 2;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float mix[S][S], out[S], in[S];
  float4 w[PER];
  bool ok[PER];
  int at[PER];
#pragma unroll
  for (int q = 0; q < PER; ++q) { at[q] = 4 * (q * nt + tid); ok[q] = q * nt + tid < n4; }
  // what no kernel of the step writes is read before the wait
#pragma unroll
  for (int t = 0; t < S; ++t) {
    in[t] = p.in ? p.in[t] : 1.f;
    out[t] = p.mix ? p.out[t] : 0.f;
#pragma unroll
    for (int s = 0; s < S; ++s) mix[s][t] = p.mix ? p.mix[s * S + t] : (s == t ? 1.f : 0.f);
  }
#pragma unroll
  for (int q = 0; q < PER; ++q) w[q] = ok[q] ? hs_load4(p.w + at[q]) : zero;
  pdl_wait();
  const int i = blockIdx.x;
  const size_t src = (size_t)(p.rows ? p.rows[i] : i);
  float4 x[S][PER], y[PER], u[PER];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    const float* xs = p.x + (p.same ? src : src * S + s) * p.hidden;
#pragma unroll
    for (int q = 0; q < PER; ++q) x[s][q] = ok[q] ? ((p.same && s > 0) ? x[0][q] : hs_load4(xs + at[q])) : zero;
  }
#pragma unroll
  for (int q = 0; q < PER; ++q) y[q] = zero;
  if (p.y) {
    const TY* yr = (const TY*)p.y + src * p.hidden;
#pragma unroll
    for (int q = 0; q < PER; ++q) if (ok[q]) y[q] = hs_load4(yr + at[q]);
  } else if (p.e) {
    for (int k0 = 0; k0 < p.top; k0 += 4) {          // four choices' rows in flight at a time, added in order
      float wk[4];
      float4 r[4][PER];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const bool have = k0 + c < p.top;
        const size_t pair = src * p.top + k0 + (have ? c : 0);
        const float* e = p.e + (size_t)p.place_of[pair] * p.hidden;
        wk[c] = have ? (p.weights ? p.weights[pair] : p.weight) : 0.f;
#pragma unroll
        for (int q = 0; q < PER; ++q) r[c][q] = ok[q] && have ? hs_load4(e + at[q]) : zero;
      }
#pragma unroll
      for (int c = 0; c < 4; ++c)
#pragma unroll
        for (int q = 0; q < PER; ++q) y[q] = hs_fma(wk[c], r[c][q], y[q]);
    }
  }
#pragma unroll
  for (int q = 0; q < PER; ++q) u[q] = zero;
#pragma unroll
  for (int t = 0; t < S; ++t) {
    float* xn = p.x_new ? p.x_new + (src * S + t) * p.hidden : nullptr;
#pragma unroll
    for (int q = 0; q < PER; ++q) {
      float4 v = x[t][q];
      if (p.mix) {
        v = zero;
#pragma unroll
        for (int s = 0; s < S; ++s) v = hs_fma(mix[s][t], x[s][q], v);
        v = hs_fma(out[t], y[q], v);
      }
      if (xn && ok[q]) hs_store4(xn + at[q], v);
      u[q] = hs_fma(in[t], v, u[q]);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int q = 0; q < PER; ++q) ss += u[q].x * u[q].x + u[q].y * u[q].y + u[q].z * u[q].z + u[q].w * u[q].w;
  const float f = rsqrtf(block_sum(ss, scratch) / (float)p.hidden + p.eps);
  TO* o = (TO*)p.normed + (size_t)i * p.hidden;
#pragma unroll
  for (int q = 0; q < PER; ++q)
    if (ok[q]) hs_store4(o + at[q], make_float4(u[q].x * f * w[q].x, u[q].y * f * w[q].y, u[q].z * f * w[q].z, u[q].w * f * w[q].w));
}

// Any number of streams and any row length: an element at a time, a column of the streams in shared memory.
template <typename TY, typename TO>
__global__ void streams_any_kernel(StreamsParams p) {
  extern __shared__ float col[];               // [S][threads]
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x, S = p.streams, nt = blockDim.x, tid = threadIdx.x;
  const size_t src = (size_t)(p.rows ? p.rows[i] : i);
  auto u_of = [&](int j, bool first) -> float {
    // the second pass reads what the first one wrote, where it wrote anything
    const bool read_new = !first && p.x_new != nullptr;
    for (int s = 0; s < S; ++s)
      col[s * nt + tid] = read_new ? p.x_new[(src * S + s) * p.hidden + j] : p.x[(p.same ? src : src * S + s) * p.hidden + j];
    float y = 0.f, u = 0.f;
    if (!read_new && p.mix) {
      if (p.y) y = to_f32(((const TY*)p.y)[src * p.hidden + j]);
      else if (p.e)
        for (int k = 0; k < p.top; ++k) {
          const size_t pair = src * p.top + k;
          y = fmaf(p.weights ? p.weights[pair] : p.weight, p.e[(size_t)p.place_of[pair] * p.hidden + j], y);
        }
    }
    for (int t = 0; t < S; ++t) {
      float v = col[t * nt + tid];
      if (!read_new && p.mix) {
        v = 0.f;
        for (int s = 0; s < S; ++s) v = fmaf(p.mix[s * S + t], col[s * nt + tid], v);
        v = fmaf(p.out[t], y, v);
      }
      if (first && p.x_new) p.x_new[(src * S + t) * p.hidden + j] = v;
      u = fmaf(p.in ? p.in[t] : 1.f, v, u);
    }
    return u;
  };
  float ss = 0.f;
  for (int j = tid; j < p.hidden; j += nt) { const float u = u_of(j, true); ss += u * u; }
  const float f = rsqrtf(block_sum(ss, scratch) / (float)p.hidden + p.eps);
  TO* o = (TO*)p.normed + (size_t)i * p.hidden;
  for (int j = tid; j < p.hidden; j += nt) o[j] = from_f32<TO>(u_of(j, false) * f * p.w[j]);
}

template <typename TY, typename TO>
int launch_streams(const StreamsParams& p, int num_rows, bool vec, cudaStream_t stream) {
  const int n4 = p.hidden >> 2;
  const int per = n4 <= 1024 ? 1 : 2;
  const int threads = ((n4 + per - 1) / per + 31) / 32 * 32;
  if (vec && threads <= 1024 && p.streams <= 4) {
#define LB_HS(S_) do { if (per == 1) launch(streams_row_kernel<TY, TO, S_, 1>, dim3(num_rows), dim3(threads), 0, stream, p); \
                       else launch(streams_row_kernel<TY, TO, S_, 2>, dim3(num_rows), dim3(threads), 0, stream, p); } while (0)
    switch (p.streams) {
      case 1: LB_HS(1); break;
      case 2: LB_HS(2); break;
      case 3: LB_HS(3); break;
      default: LB_HS(4); break;
    }
#undef LB_HS
    return 0;
  }
  int t = p.hidden >= 2048 ? 512 : (p.hidden >= 512 ? 256 : 64);
  while (t > 32 && (size_t)t * p.streams * sizeof(float) > 40 * 1024) t /= 2;
  launch(streams_any_kernel<TY, TO>, dim3(num_rows), dim3(t), (size_t)t * p.streams * sizeof(float), stream, p);
  return 0;
}

}  // namespace lb

// One row for each of num_rows (rows[i] of the operands if `rows` is given; the streams are then not written).  y_dtype: the type
// of y.  With mix: out, and either y or the experts' e with place_of.
LB_EXPORT int lb_streams_norm(void* normed, int out_dtype, const float* x, float* x_new, int streams, int same, const float* mix,
                              const float* out, const float* in, const void* y, int y_dtype, const float* e, const int* place_of,
                              const float* weights, int top, float weight, const float* w, float eps, const int* rows, int num_rows,
                              int hidden, cudaStream_t stream) {
  LB_CHECK_ARG(lb::valid_dtype(out_dtype) && lb::valid_dtype(y_dtype), "streams_norm: bad dtype");
  LB_CHECK_ARG(normed && x && w && num_rows >= 0 && hidden > 0, "streams_norm: bad arguments");
  LB_CHECK_ARG(streams > 0 && streams <= 256, "streams_norm: %d streams, at most 256", streams);
  LB_CHECK_ARG(mix ? (out != nullptr && ((y != nullptr) != (e != nullptr))) : (!out && !y && !e && !x_new),
               "streams_norm: a mix goes with a sublayer's output, and only with it do the streams change");
  LB_CHECK_ARG(!e || (place_of && top > 0), "streams_norm: experts' rows need the pairs' places");
  LB_CHECK_ARG(!(rows && x_new), "streams_norm: with a row list the streams are not written");
  LB_CHECK_ARG(!(same && x_new == x && streams > 1), "streams_norm: one row for all streams cannot be updated in place");
  if (num_rows == 0) return 0;
  lb::StreamsParams p;
  p.normed = normed; p.x = x; p.x_new = x_new; p.streams = streams; p.same = same; p.mix = mix; p.out = out; p.in = in; p.y = y;
  p.e = e; p.place_of = place_of; p.weights = weights; p.top = top; p.weight = weight; p.w = w; p.eps = eps; p.rows = rows; p.hidden = hidden;
  auto al = [](const void* ptr) { return (uintptr_t)ptr % 16 == 0; };
  const bool vec = hidden % 4 == 0 && al(normed) && al(x) && al(x_new) && al(y) && al(e) && al(w);
  LB_DISPATCH_DTYPE(y_dtype, TY, {
    LB_DISPATCH_DTYPE(out_dtype, TO, { lb::launch_streams<TY, TO>(p, num_rows, vec, stream); })
  })
  LB_CHECK_LAUNCH("streams_norm");
  return 0;
}
