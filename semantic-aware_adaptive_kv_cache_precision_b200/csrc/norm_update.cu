// The step between two sublayers of a layer that norms a sublayer's OUTPUT (and nothing
// else) before it joins the fp32 residual stream:
//
//   x += y / sqrt(mean(y^2) + eps) * (add_offset + w_add)        (y: the sublayer's output)
//   out = x, in the type the next sublayer reads                  (w_out null)
//   out = x / sqrt(mean(x^2) + eps) * (out_offset + w_out)       (w_out given: a norm)
//
// one pass over the stream. Any of the three may be absent: without y nothing is added (the
// copy of the stream for a first layer, or a plain RMS norm with a weight stored around zero,
// `offset` 1, or around one, `offset` 0); without out only the stream is completed. With
// `rows` only those rows are normed or copied (the final norm of the wanted positions). Sums
// of squares, roots and products are fp32 with one rounding at the store; one block a row,
// the row in shared memory, so the order of the additions depends on the row's length alone.
//
// `rms_join` is the step of a layer whose norm comes AFTER the sum:
//
//   x <- v / sqrt(mean(v^2) + eps) * w,   v = alpha x + scale (n_a(y_a) + n_b(y_b))
//   out = x in the type the next sublayer reads
//
// with n(y) = y, or y / sqrt(mean(y^2) + branch_eps) * w_branch where a sublayer is two mixers
// side by side whose outputs are normed before they are summed (y_b may be absent).
#include "common.cuh"

namespace {

constexpr int kThreads = 256;

__device__ __forceinline__ float inverse_rms(const float* row, int hidden, float eps,
                                             float* scratch) {
  float q = 0.f;
  for (int i = threadIdx.x; i < hidden; i += kThreads) q = fmaf(row[i], row[i], q);
  return 1.f / sqrtf(block_sum(q, scratch) / static_cast<float>(hidden) + eps);
}

template <typename W, typename Out>
__global__ void __launch_bounds__(kThreads)
rms_update_kernel(float* __restrict__ x, const float* __restrict__ y,
                  const W* __restrict__ w_add, float add_offset,
                  const int32_t* __restrict__ rows, const W* __restrict__ w_out, float out_offset,
                  Out* __restrict__ out, int hidden, float eps) {
  extern __shared__ float row[];
  __shared__ float scratch[33];
  const long long src = rows ? rows[blockIdx.x] : blockIdx.x;
  float* in = x + src * hidden;
  if (y != nullptr) {
    const float* add = y + src * hidden;
    for (int i = threadIdx.x; i < hidden; i += kThreads) row[i] = add[i];
    __syncthreads();
    const float r = inverse_rms(row, hidden, eps, scratch);
    for (int i = threadIdx.x; i < hidden; i += kThreads) {
      const float v = in[i] + row[i] * r * (add_offset + widen(w_add[i]));
      in[i] = v;
      row[i] = v;
    }
  } else {
    for (int i = threadIdx.x; i < hidden; i += kThreads) row[i] = in[i];
  }
  if (out == nullptr) return;
  Out* o = out + (long long)blockIdx.x * hidden;
  if (w_out == nullptr) {                   // (each thread reads back what it wrote itself)
    for (int i = threadIdx.x; i < hidden; i += kThreads) o[i] = narrow<Out>(row[i]);
    return;
  }
  __syncthreads();
  const float r = inverse_rms(row, hidden, eps, scratch);
  for (int i = threadIdx.x; i < hidden; i += kThreads)
    o[i] = narrow<Out>(row[i] * r * (out_offset + widen(w_out[i])));
}

template <typename W, typename Out>
int launch(float* x, const float* y, const void* w_add, float add_offset, const int32_t* rows,
           const void* w_out, float out_offset, void* out, int n, int hidden, float eps,
           cudaStream_t stream) {
  return launch_ordered(rms_update_kernel<W, Out>, dim3(n), dim3(kThreads),
                        (size_t)hidden * sizeof(float), stream, x, y, (const W*)w_add, add_offset,
                        rows, (const W*)w_out, out_offset, (Out*)out, hidden, eps);
}

// One block a row; a thread keeps its four-wide pieces of the row in registers (VEC: the row's
// length is a multiple of four, NV pieces a thread at most), all loads of the row go out
// together, and the two branches' sums of squares are taken in one reduction.
__device__ __forceinline__ float2 block_sum2(float2 v, float2* scratch /* >= 33 */) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
  v.x = warp_sum(v.x);
  v.y = warp_sum(v.y);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float2 total = make_float2(0.f, 0.f);
  for (int w = 0; w < warps; ++w) {
    total.x += scratch[w].x;
    total.y += scratch[w].y;
  }
  return total;
}

template <typename W>
__device__ __forceinline__ float4 widen4(const W* p);
template <>
__device__ __forceinline__ float4 widen4<float>(const float* p) {
  return *reinterpret_cast<const float4*>(p);
}
template <>
__device__ __forceinline__ float4 widen4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 r[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<uint2*>(r);
}
__device__ __forceinline__ float dot4(float4 a) {
  return fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, a.w * a.w)));
}

template <int NV, typename W, typename Out>
__global__ void rms_join_vec_kernel(float* __restrict__ x, const float* __restrict__ ya,
                                    const W* __restrict__ wa, const float* __restrict__ yb,
                                    const W* __restrict__ wb, float branch_eps, float scale,
                                    float alpha, const W* __restrict__ w, float eps,
                                    Out* __restrict__ out, int hidden) {
  __shared__ float2 scratch[33];
  const long long base = (long long)blockIdx.x * hidden;
  float4 v[NV], a[NV], b[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    v[i] = a[i] = b[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c >= hidden) continue;
    v[i] = *reinterpret_cast<const float4*>(x + base + c);
    a[i] = *reinterpret_cast<const float4*>(ya + base + c);
    if (yb) b[i] = *reinterpret_cast<const float4*>(yb + base + c);
  }
  float ra = 1.f, rb = 1.f;
  if (wa) {
    float2 ss = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      ss.x += dot4(a[i]);
      ss.y += dot4(b[i]);
    }
    ss = block_sum2(ss, scratch);
    ra = 1.f / sqrtf(ss.x / static_cast<float>(hidden) + branch_eps);
    rb = 1.f / sqrtf(ss.y / static_cast<float>(hidden) + branch_eps);
  }
  float2 q = make_float2(0.f, 0.f);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    if (c >= hidden) continue;
    float4 s = a[i];
    if (wa) {
      const float4 k = widen4<W>(wa + c);
      s.x *= ra * k.x; s.y *= ra * k.y; s.z *= ra * k.z; s.w *= ra * k.w;
    }
    if (yb) {
      const float4 k = wb ? widen4<W>(wb + c) : make_float4(1.f, 1.f, 1.f, 1.f);
      s.x = fmaf(b[i].x, rb * k.x, s.x); s.y = fmaf(b[i].y, rb * k.y, s.y);
      s.z = fmaf(b[i].z, rb * k.z, s.z); s.w = fmaf(b[i].w, rb * k.w, s.w);
    }
    v[i].x = fmaf(alpha, v[i].x, scale * s.x); v[i].y = fmaf(alpha, v[i].y, scale * s.y);
    v[i].z = fmaf(alpha, v[i].z, scale * s.z); v[i].w = fmaf(alpha, v[i].w, scale * s.w);
    q.x += dot4(v[i]);
  }
  q = block_sum2(q, scratch);
  const float r = 1.f / sqrtf(q.x / static_cast<float>(hidden) + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    if (c >= hidden) continue;
    const float4 k = widen4<W>(w + c);
    const float4 o = make_float4(v[i].x * r * k.x, v[i].y * r * k.y, v[i].z * r * k.z,
                                 v[i].w * r * k.w);
    store4(x + base + c, o);
    if (out) store4(out + base + c, o);
  }
}

// The same for rows of any length, the summed row in shared memory.
template <typename W, typename Out>
__global__ void __launch_bounds__(kThreads)
rms_join_kernel(float* __restrict__ x, const float* __restrict__ ya, const W* __restrict__ wa,
                const float* __restrict__ yb, const W* __restrict__ wb, float branch_eps,
                float scale, float alpha, const W* __restrict__ w, float eps,
                Out* __restrict__ out, int hidden) {
  extern __shared__ float row[];
  __shared__ float scratch[33];
  const long long base = (long long)blockIdx.x * hidden;
  float ra = 1.f, rb = 1.f;
  if (wa) {
    ra = inverse_rms(ya + base, hidden, branch_eps, scratch);
    if (yb) rb = inverse_rms(yb + base, hidden, branch_eps, scratch);
  }
  for (int i = threadIdx.x; i < hidden; i += kThreads) {
    float s = ya[base + i];
    if (wa) s *= ra * widen(wa[i]);
    if (yb) s = fmaf(yb[base + i], wb ? rb * widen(wb[i]) : 1.f, s);
    row[i] = fmaf(alpha, x[base + i], scale * s);
  }
  const float r = inverse_rms(row, hidden, eps, scratch);   // (a thread reads its own numbers)
  for (int i = threadIdx.x; i < hidden; i += kThreads) {
    const float o = row[i] * r * widen(w[i]);
    x[base + i] = o;
    if (out) out[base + i] = narrow<Out>(o);
  }
}

template <typename W, typename Out>
int launch_join(float* x, const float* ya, const void* wa, const float* yb, const void* wb,
                float branch_eps, float scale, float alpha, const void* w, float eps, void* out,
                int n, int hidden, cudaStream_t stream) {
  const uintptr_t all = (uintptr_t)x | (uintptr_t)ya | (uintptr_t)yb | (uintptr_t)wa |
                        (uintptr_t)wb | (uintptr_t)w | (uintptr_t)out;
  if (hidden % 4 == 0 && hidden <= 4 * 4 * 512 && !(all & 15)) {
    const int pieces = hidden / 4;
    const int nv = pieces <= 256 ? 1 : pieces <= 1024 ? 2 : 4;
    const int threads = ((pieces + nv - 1) / nv + 31) / 32 * 32;
#define SAKV_JOIN(NV)                                                                            \
  return launch_ordered(rms_join_vec_kernel<NV, W, Out>, dim3(n), dim3(threads), 0, stream, x,   \
                        ya, (const W*)wa, yb, (const W*)wb, branch_eps, scale, alpha,            \
                        (const W*)w, eps, (Out*)out, hidden)
    if (nv == 1) SAKV_JOIN(1);
    if (nv == 2) SAKV_JOIN(2);
    SAKV_JOIN(4);
#undef SAKV_JOIN
  }
  return launch_ordered(rms_join_kernel<W, Out>, dim3(n), dim3(kThreads),
                        (size_t)hidden * sizeof(float), stream, x, ya, (const W*)wa, yb,
                        (const W*)wb, branch_eps, scale, alpha, (const W*)w, eps, (Out*)out,
                        hidden);
}

}  // namespace

// x: fp32 [n, hidden], replaced by the norm (weight w) of alpha x + scale (n(ya) + n(yb)); ya,
// yb: fp32 [n, hidden] (yb null: none); wa, wb [hidden]: the branches' norm weights (null: as
// they are; both or neither where there are two). Weights of `w_dtype`. out (null: none): x in
// `out_dtype`.
SAKV_EXPORT int sakv_rms_join(float* x, const float* ya, const void* wa, const float* yb,
                              const void* wb, float branch_eps, float scale, float alpha,
                              const void* w, int w_dtype, float eps, void* out, int out_dtype,
                              int n, int hidden, cudaStream_t stream) {
  if (n < 0 || hidden <= 0 || hidden > 12000 || !ya || !w || (yb && (!wa != !wb)) || (!yb && wb))
    return cudaErrorInvalidValue;
  if (n == 0) return 0;
#define SAKV_J(W, O)                                                                             \
  return launch_join<W, O>(x, ya, wa, yb, wb, branch_eps, scale, alpha, w, eps, out, n, hidden,  \
                           stream)
  if (w_dtype == SAKV_F32 && out_dtype == SAKV_F32) SAKV_J(float, float);
  if (w_dtype == SAKV_BF16 && out_dtype == SAKV_BF16) SAKV_J(__nv_bfloat16, __nv_bfloat16);
  if (w_dtype == SAKV_BF16 && out_dtype == SAKV_F32) SAKV_J(__nv_bfloat16, float);
  if (w_dtype == SAKV_F32 && out_dtype == SAKV_BF16) SAKV_J(float, __nv_bfloat16);
#undef SAKV_J
  return cudaErrorInvalidValue;
}

// x: fp32 [T, hidden], updated in place when `y` (fp32 [T, hidden]) is given. out (may be
// null): [n, hidden] of `out_dtype`, the rows `rows ? rows[r] : r`; `rows` only without `y`.
// Weights of `w_dtype`.
SAKV_EXPORT int sakv_rms_update(float* x, const float* y, const void* w_add, float add_offset,
                                const int32_t* rows, const void* w_out, float out_offset,
                                int w_dtype, void* out, int out_dtype, int n, int hidden,
                                float eps, cudaStream_t stream) {
  if (n < 0 || hidden <= 0 || hidden > 12000 || (y != nullptr && (rows != nullptr || !w_add)) ||
      (out == nullptr && y == nullptr))
    return cudaErrorInvalidValue;
  if (n == 0) return 0;
  if (w_dtype == SAKV_F32 && out_dtype == SAKV_F32)
    return launch<float, float>(x, y, w_add, add_offset, rows, w_out, out_offset, out, n, hidden,
                                eps, stream);
  if (w_dtype == SAKV_BF16 && out_dtype == SAKV_BF16)
    return launch<__nv_bfloat16, __nv_bfloat16>(x, y, w_add, add_offset, rows, w_out, out_offset,
                                                out, n, hidden, eps, stream);
  if (w_dtype == SAKV_BF16 && out_dtype == SAKV_F32)
    return launch<__nv_bfloat16, float>(x, y, w_add, add_offset, rows, w_out, out_offset, out, n,
                                        hidden, eps, stream);
  if (w_dtype == SAKV_F32 && out_dtype == SAKV_BF16)
    return launch<float, __nv_bfloat16>(x, y, w_add, add_offset, rows, w_out, out_offset, out, n,
                                        hidden, eps, stream);
  return cudaErrorInvalidValue;
}
