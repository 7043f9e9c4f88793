// The gated delta rule: a recurrence with a matrix of state a head, which fades by one number a
// head and token and whose read-out along the current unit key is corrected towards the value:
//
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q          (S: dim x vdim, fp32)
//
// with q and k (kv_heads of them; head h reads head floor(h / (heads / kv_heads))) and v each
// through a short causal convolution a channel and silu, q and k unit vectors a head (q times a
// constant), g = exp(-exp(A_log) softplus(a + dt_bias)) and beta = sigmoid(b), a number a head.
//
// Two kernels. `delta_inputs` works out what does not depend on the state, four consecutive tokens
// of a sequence to a warp: convolutions, silu, unit vectors, decays and betas, all fp32. The scan
// is the recurrence: a block owns some neighbouring value columns of one head of one sequence, a
// column's rows are dealt to RS neighbouring lanes (four neighbouring rows at a time, RP rows a
// lane), the state stays in registers, and the tokens' q, k, v arrive in shared memory by cp.async
// a chunk ahead. It comes in two forms:
//
//   * `delta_walk` takes one token at a time. Its sums have the same terms in the same order
//     however the tokens are cut into steps.
//   * `delta_groups` takes four tokens at a time (prompts in the 16-bit mode). Within a group the
//     recurrence is unrolled: with c_i the decay from the group's start to token i and S the state
//     at its start,
//         u_i = beta_i (v_i - c_i S^T k_i - sum_{j<i} (c_i / c_j) (k_j . k_i) u_j)
//         o_i = c_i S^T q_i + sum_{j<=i} (c_i / c_j) (k_j . q_i) u_j
//         S  <- c_3 S + sum_j (c_3 / c_j) k_j u_j^T
//     so that the eight sums over a column (four keys, four queries) are taken from the SAME state
//     and cross the lanes together, once every four tokens instead of twice every token. The
//     products k.k and k.q and the factors made of them and of the decays are the same for all
//     columns: `delta_inputs` leaves them as 40 numbers a (group, head). All of it is fp32.
//
// The state is moved by its change (S + (g - 1) S, with g - 1 = expm1 of the logarithm), so a decay
// close to 1 keeps its distance from 1.
#include "common.cuh"

namespace {

constexpr int kGroup = 4;              // tokens of a group
constexpr int kCoef = 40;              // numbers a (group, head)
constexpr int kChunk = 16;             // tokens brought into shared memory at a time
constexpr int kTwoWarps = 3;           // warps an SM from which on a thread takes two columns
// places among a group's numbers: beta; beta c; c; the decay from each token to the group's end;
// the rows of (c_i / c_j) (k_j . q_i); beta_i (c_i / c_j) (k_j . k_i) for (i, j) = (1, 0), (2, 0),
// (2, 1), (3, 0), (3, 1), (3, 2); the whole group's decay less one
constexpr int kBeta = 0, kBetaC = 4, kC = 8, kEnd = 12, kOut = 16, kSolve = 32, kFade = 38;

__device__ __forceinline__ float silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// Where a sequence's groups begin among all groups of the step (never two in one place: a
// sequence of n tokens has at most floor(n / 4) + 1 groups).
__device__ __forceinline__ long long first_group(const int32_t* cu_seqlens, int b) {
  return cu_seqlens[b] / kGroup + b;
}

template <typename W>
struct DeltaInputs {
  const float* proj;                   // [tokens, stride]: q, k, v (the convolution's input) first
  long long stride;
  int a_off, b_off;                    // a column a head each
  const W* conv;                       // [channels, taps]
  const float* a;                      // [heads]: -exp(A_log)
  const float* dt_bias;                // [heads]
  float* conv_state;                   // [slots, taps - 1, channels]
  const int32_t* cu_seqlens;
  const int32_t* slots;
  float* prepared;                     // [tokens, channels]: unit q, unit k, v
  float* gates;                        // [tokens, heads, 2]: decay less one, beta
  float* coef;                         // [groups, heads, kCoef], or null
  int heads, kv_heads, dim, vdim, taps, channels, move_state;
  float q_scale, unit_eps;
};

// silu of the convolution of one channel for the group's `m` tokens; token tt is number i0 + tt of
// its sequence's part in this step. Inputs before the part come from the sequence's running ones.
// TAPS: the taps as a compile-time number, so that the window of inputs is read once for all four
// tokens (0: any number). The products are added oldest first either way.
template <int TAPS, typename W>
__device__ __forceinline__ void conv_channel(const DeltaInputs<W>& p, const float* __restrict__ part,
                                             const float* __restrict__ old, int c, int i0, int m,
                                             float (&y)[kGroup]) {
  const int taps = TAPS > 0 ? TAPS : p.taps, keep = taps - 1;
  auto input = [&](int at) {                           // input number `at` of this step's part
    return at >= 0 ? __ldg(part + (long long)at * p.stride + c)
                   : __ldg(old + (long long)(keep + at) * p.channels + c);
  };
#pragma unroll
  for (int tt = 0; tt < kGroup; ++tt) y[tt] = 0.f;
  if constexpr (TAPS > 0) {
    float x[TAPS - 1 + kGroup], w[TAPS];
#pragma unroll
    for (int i = 0; i < TAPS - 1 + kGroup; ++i) x[i] = i < keep + m ? input(i0 - keep + i) : 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = widen(p.conv[(long long)c * TAPS + j]);
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int tt = 0; tt < kGroup; ++tt) y[tt] = fmaf(x[tt + j], w[j], y[tt]);
  } else {
    for (int j = 0; j < taps; ++j) {
      const float w = widen(p.conv[(long long)c * taps + j]);
#pragma unroll
      for (int tt = 0; tt < kGroup; ++tt)
        if (tt < m) y[tt] = fmaf(input(i0 + tt - (keep - j)), w, y[tt]);
    }
  }
#pragma unroll
  for (int tt = 0; tt < kGroup; ++tt) y[tt] = silu(y[tt]);
}

// Grid: (units of warps, sequences). A group's units are its kv_heads (q and k of one head, with
// the decays, betas and group numbers of the heads that read it), then runs of 32 * PER channels
// of v. PER * 32 >= dim.
template <int PER, int TAPS, typename W>
__global__ void __launch_bounds__(128) delta_inputs_kernel(const DeltaInputs<W> p) {
  let_next_kernel_start();
  wait_for_previous_kernel();
  const int b = blockIdx.y, lane = threadIdx.x & 31;
  const int first = p.cu_seqlens[b], n = p.cu_seqlens[b + 1] - first;
  const int v_width = p.heads * p.vdim;
  const int units = p.kv_heads + (v_width + 32 * PER - 1) / (32 * PER);
  const long long warp = blockIdx.x * (long long)(blockDim.x >> 5) + (threadIdx.x >> 5);
  const int group = static_cast<int>(warp / units), unit = static_cast<int>(warp - (long long)group * units);
  const int i0 = group * kGroup;
  if (i0 >= n) return;
  const int m = n - i0 < kGroup ? n - i0 : kGroup;
  const float* part = p.proj + (long long)first * p.stride;
  const float* old = p.conv_state + (long long)p.slots[b] * (p.taps - 1) * p.channels;
  float* __restrict__ out = p.prepared + (long long)(first + i0) * p.channels;
  const int qk = p.kv_heads * p.dim;

  if (unit >= p.kv_heads) {                            // values: the convolution is all
    const int c0 = (unit - p.kv_heads) * 32 * PER;
    float y[PER][kGroup];
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int c = c0 + lane + 32 * i;
      if (c < v_width) conv_channel<TAPS>(p, part, old, 2 * qk + c, i0, m, y[i]);
    }
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int c = c0 + lane + 32 * i;
#pragma unroll
      for (int tt = 0; tt < kGroup; ++tt)
        if (tt < m && c < v_width) out[(long long)tt * p.channels + 2 * qk + c] = y[i][tt];
    }
    return;
  }

  float q[PER][kGroup], k[PER][kGroup];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = lane + 32 * i, c = unit * p.dim + e;
#pragma unroll
    for (int tt = 0; tt < kGroup; ++tt) q[i][tt] = k[i][tt] = 0.f;
    if (e < p.dim) {
      conv_channel<TAPS>(p, part, old, c, i0, m, q[i]);
      conv_channel<TAPS>(p, part, old, qk + c, i0, m, k[i]);
    }
  }
#pragma unroll
  for (int tt = 0; tt < kGroup; ++tt) {
    if (tt >= m) {                                     // (a token that is missing: zeros)
#pragma unroll
      for (int i = 0; i < PER; ++i) q[i][tt] = k[i][tt] = 0.f;
    }
    float qq = 0.f, kk = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      qq = fmaf(q[i][tt], q[i][tt], qq);
      kk = fmaf(k[i][tt], k[i][tt], kk);
    }
    const float rq = p.q_scale / sqrtf(warp_sum(qq) + p.unit_eps);
    const float rk = 1.f / sqrtf(warp_sum(kk) + p.unit_eps);
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int e = lane + 32 * i;
      q[i][tt] *= rq;
      k[i][tt] *= rk;
      if (tt < m && e < p.dim) {
        float* row = out + (long long)tt * p.channels + unit * p.dim + e;
        row[0] = q[i][tt];
        row[qk] = k[i][tt];
      }
    }
  }
  // k_j . q_i and k_j . k_i of the group
  float kq[kGroup][kGroup] = {}, kkg[kGroup][kGroup] = {};
  if (p.coef != nullptr) {
#pragma unroll
    for (int i = 0; i < kGroup; ++i)
#pragma unroll
      for (int j = 0; j <= i; ++j) {
        float s = 0.f, r = 0.f;
#pragma unroll
        for (int e = 0; e < PER; ++e) {
          s = fmaf(k[e][j], q[e][i], s);
          if (j < i) r = fmaf(k[e][j], k[e][i], r);
        }
        kq[i][j] = warp_sum(s);
        if (j < i) kkg[i][j] = warp_sum(r);
      }
  }
  // a lane a (head, token of the group)
  const int per = p.heads / p.kv_heads, i = lane & 3;
  for (int x0 = 0; x0 < per; x0 += 8) {
    const int x = x0 + (lane >> 2);
    const bool live = x < per;
    const int h = unit * per + (live ? x : 0);
    float log_g = 0.f, beta = 0.f;
    if (i < m) {
      const float* row = part + (long long)(i0 + i) * p.stride;
      log_g = softplus(row[p.a_off + h] + p.dt_bias[h]) * p.a[h];
      beta = 1.f / (1.f + expf(-row[p.b_off + h]));
      if (live) {
        float* to = p.gates + ((long long)(first + i0 + i) * p.heads + h) * 2;
        to[0] = expm1f(log_g);
        to[1] = beta;
      }
    }
    if (p.coef == nullptr) continue;
    float g[kGroup], since = 0.f, rest = 0.f, between = 0.f;
#pragma unroll
    for (int j = 0; j < kGroup; ++j) {
      g[j] = __shfl_sync(0xffffffffu, log_g, (lane & ~3) + j);
      if (j <= i) since += g[j];                        // the logarithm of c_i
      else rest += g[j];                                // from token i to the group's end
    }
    if (!live) continue;
    float* to = p.coef + ((first_group(p.cu_seqlens, b) + group) * p.heads + h) * kCoef;
    const float c = expf(since);
    to[kBeta + i] = beta;
    to[kBetaC + i] = beta * c;
    to[kC + i] = c;
    to[kEnd + i] = expf(rest);
#pragma unroll
    for (int j = kGroup - 1; j >= 0; --j) {
      if (j + 1 < kGroup && j < i) between += g[j + 1];  // the logarithm of c_i / c_j
      float along_q = kq[0][j], along_k = 0.f;
#pragma unroll
      for (int r = 1; r < kGroup; ++r)
        if (r == i) {
          along_q = kq[r][j];
          along_k = kkg[r][j];
        }
      const float d = expf(between);
      to[kOut + 4 * i + j] = j <= i ? d * along_q : 0.f;
      if (j < i) to[kSolve + i * (i - 1) / 2 + j] = beta * d * along_k;
    }
    if (i == kGroup - 1) {
      to[kFade] = expm1f(since);
      to[kFade + 1] = 0.f;
    }
  }
}

// The same for a step in which every sequence brings one token: a thread a channel, a block q and k
// of one head (with its heads' decays and betas) or blockDim channels of v. Every sum has its terms
// in the order of the kernel above. The running inputs go up by one place.
template <typename W>
__global__ void delta_inputs_step_kernel(const DeltaInputs<W> p) {
  extern __shared__ float ys[];                        // [2 dim]
  __shared__ float inv[2];
  let_next_kernel_start();
  wait_for_previous_kernel();
  const int b = blockIdx.y, unit = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const long long t = p.cu_seqlens[b];
  const int qk = p.kv_heads * p.dim, keep = p.taps - 1;
  const float* row = p.proj + t * p.stride;
  float* old = p.conv_state + (long long)p.slots[b] * keep * p.channels;
  float* out = p.prepared + t * p.channels;
  auto conv = [&](int c) {
    constexpr int kMost = 7;                           // running inputs held in registers
    const float now = row[c];
    float y = 0.f;
    if (keep <= kMost) {
      float x[kMost + 1];
#pragma unroll
      for (int j = 0; j < kMost; ++j) x[j] = j < keep ? old[(long long)j * p.channels + c] : now;
      x[kMost] = now;
#pragma unroll
      for (int j = 0; j < kMost + 1; ++j)
        if (j <= keep) y = fmaf(x[j], widen(p.conv[(long long)c * p.taps + j]), y);
      if (p.move_state) {
#pragma unroll
        for (int j = 0; j < kMost; ++j)
          if (j < keep) old[(long long)j * p.channels + c] = x[j + 1];
      }
    } else {
      for (int j = 0; j < keep; ++j)
        y = fmaf(old[(long long)j * p.channels + c], widen(p.conv[(long long)c * p.taps + j]), y);
      y = fmaf(now, widen(p.conv[(long long)c * p.taps + keep]), y);
      if (p.move_state) {
        for (int j = 0; j + 1 < keep; ++j)
          old[(long long)j * p.channels + c] = old[(long long)(j + 1) * p.channels + c];
        old[(long long)(keep - 1) * p.channels + c] = now;
      }
    }
    return silu(y);
  };
  if (unit >= p.kv_heads) {
    const int c = (unit - p.kv_heads) * blockDim.x + threadIdx.x;
    if (c < p.heads * p.vdim) out[2 * qk + c] = conv(2 * qk + c);
    return;
  }
  const int e = threadIdx.x;
  const bool mine = e < 2 * p.dim, is_k = e >= p.dim;
  const int c = (is_k ? qk - p.dim : 0) + unit * p.dim + e;
  float y = 0.f;
  if (mine) ys[e] = y = conv(c);
  if (warp == 3) {                                     // (a block has four warps at least)
    const int per = p.heads / p.kv_heads;
    for (int x = lane; x < per; x += 32) {
      const int h = unit * per + x;
      float* to = p.gates + (t * p.heads + h) * 2;
      to[0] = expm1f(softplus(row[p.a_off + h] + p.dt_bias[h]) * p.a[h]);
      to[1] = 1.f / (1.f + expf(-row[p.b_off + h]));
    }
  }
  __syncthreads();
  if (warp < 2) {
    float s = 0.f;
    for (int i = lane; i < p.dim; i += 32) s = fmaf(ys[warp * p.dim + i], ys[warp * p.dim + i], s);
    s = warp_sum(s);
    if (lane == 0) inv[warp] = (warp == 0 ? p.q_scale : 1.f) / sqrtf(s + p.unit_eps);
  }
  __syncthreads();
  if (mine) out[c] = y * inv[is_k];
}

__device__ __forceinline__ void copy16_async(float* dst, const float* src) {
  const uint32_t to = static_cast<uint32_t>(__cvta_generic_to_shared(dst));
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(to), "l"(src) : "memory");
}

struct DeltaScan {
  const float* prepared;               // [tokens, channels]
  const float* gates;                  // [tokens, heads, 2]
  const float* coef;                   // [groups, heads, kCoef] (the form with groups)
  float* state;                        // [slots, heads, vdim, dim]: a column's rows lie together
  const int32_t* cu_seqlens;
  const int32_t* slots;
  float* out;                          // [tokens, heads * vdim]
  int heads, kv_heads, dim, vdim, channels, cols, chunk, keep_state;
};

// A block's share of the recurrence: its state in registers, and the copies of its tokens' inputs.
// Row p * RS * 4 + r * 4 + i of a column is number 4 p + i of lane r; rows from `dim` on are zeros.
// CV neighbouring columns belong to one thread.
template <int RP, int RS, int CV>
struct Columns {
  static constexpr int kRows = RP * RS;
  const DeltaScan& p;
  int h, b, col0, r, j, first, last, slot;
  float s[CV][RP];

  __device__ __forceinline__ Columns(const DeltaScan& p_) : p(p_) {
    h = blockIdx.y;
    b = blockIdx.z;
    col0 = blockIdx.x * p.cols;
    r = threadIdx.x % RS;
    j = threadIdx.x / RS * CV;
    first = p.cu_seqlens[b];
    last = p.cu_seqlens[b + 1];
    slot = p.slots[b];
  }
  __device__ __forceinline__ bool live(int c) const { return col0 + j + c < p.vdim; }
  __device__ __forceinline__ float* home(int c) const {
    return p.state + (((long long)slot * p.heads + h) * p.vdim + col0 + (live(c) ? j + c : 0)) * p.dim;
  }
  __device__ __forceinline__ void load() {
#pragma unroll
    for (int c = 0; c < CV; ++c) {
      const float* from = home(c);
#pragma unroll
      for (int k = 0; k < RP; k += 4) {
        const int row = k * RS + r * 4;
        float* to = s[c] + k;
        if (live(c) && p.dim % 4 == 0 && row < p.dim) {
          const float4 v = *reinterpret_cast<const float4*>(from + row);
          to[0] = v.x; to[1] = v.y; to[2] = v.z; to[3] = v.w;
        } else {
#pragma unroll
          for (int i = 0; i < 4; ++i) to[i] = live(c) && row + i < p.dim ? from[row + i] : 0.f;
        }
      }
    }
  }
  __device__ __forceinline__ void store() const {
#pragma unroll
    for (int c = 0; c < CV; ++c) {
      if (!live(c)) continue;
      float* to = home(c);
#pragma unroll
      for (int k = 0; k < RP; k += 4) {
        const int row = k * RS + r * 4;
        const float* from = s[c] + k;
        if (p.dim % 4 == 0 && row < p.dim) {
          *reinterpret_cast<float4*>(to + row) = make_float4(from[0], from[1], from[2], from[3]);
        } else {
#pragma unroll
          for (int i = 0; i < 4; ++i)
            if (row + i < p.dim) to[row + i] = from[i];
        }
      }
    }
  }
  // a buffer: q [chunk, kRows], k [chunk, kRows], v [chunk, cols], then the tokens' gates or the
  // groups' numbers
  __device__ __forceinline__ int floats(int extra) const {
    return p.chunk * (2 * kRows + p.cols) + extra;
  }
  // Brings `count` tokens from token t0 on (whole rows of zeros up to a multiple of `round`).
  __device__ __forceinline__ void fetch(float* buffer, int t0, int count, int round) const {
    const int padded = (count + round - 1) / round * round;
    const int group = p.heads / p.kv_heads;
    const int q_off = h / group * p.dim, k_off = q_off + p.kv_heads * p.dim;
    const int v_off = 2 * p.kv_heads * p.dim + h * p.vdim + col0;
    float* qs = buffer;
    float* ks = qs + p.chunk * kRows;
    float* vs = ks + p.chunk * kRows;
    const float* rows = p.prepared + (long long)t0 * p.channels;
    constexpr int kQuads = kRows / 4;
    const bool wide = p.dim % 4 == 0 && p.vdim % 4 == 0 && p.cols % 4 == 0;
    for (int e = threadIdx.x; e < padded * kQuads; e += blockDim.x) {
      const int tt = e / kQuads, i = (e - tt * kQuads) * 4;
      const float* row = rows + (long long)tt * p.channels + i;
      float* dq = qs + tt * kRows + i;
      float* dk = ks + tt * kRows + i;
      if (wide && tt < count && i < p.dim) {
        copy16_async(dq, row + q_off);
        copy16_async(dk, row + k_off);
      } else {
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          const bool real = tt < count && i + n < p.dim;
          dq[n] = real ? row[q_off + n] : 0.f;
          dk[n] = real ? row[k_off + n] : 0.f;
        }
      }
    }
    if (wide) {
      const int quads = p.cols / 4;
      for (int e = threadIdx.x; e < padded * quads; e += blockDim.x) {
        const int tt = e / quads, i = (e - tt * quads) * 4;
        float* to = vs + tt * p.cols + i;
        if (tt < count && col0 + i < p.vdim)
          copy16_async(to, rows + (long long)tt * p.channels + v_off + i);
        else
          *reinterpret_cast<float4*>(to) = make_float4(0.f, 0.f, 0.f, 0.f);
      }
    } else {
      for (int e = threadIdx.x; e < padded * p.cols; e += blockDim.x) {
        const int tt = e / p.cols, i = e - tt * p.cols;
        vs[e] = tt < count && col0 + i < p.vdim ? rows[(long long)tt * p.channels + v_off + i] : 0.f;
      }
    }
  }
};

__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void copies_wait_all_but_last() {
  asm volatile("cp.async.wait_group 1;" ::: "memory");
}

// One token at a time.
template <int RP, int RS>
__global__ void __launch_bounds__(256) delta_walk_kernel(const DeltaScan p) {
  extern __shared__ __align__(16) float shared[];
  let_next_kernel_start();
  wait_for_previous_kernel();
  Columns<RP, RS, 1> c(p);
  const int per_buffer = c.floats(2 * p.chunk);
  constexpr int kRows = RP * RS;
  auto fetch = [&](int t0, int buffer) {
    const int count = min(p.chunk, c.last - t0);
    float* to = shared + buffer * per_buffer;
    c.fetch(to, t0, count, 1);
    float* gs = to + p.chunk * (2 * kRows + p.cols);
    for (int e = threadIdx.x; e < 2 * count; e += blockDim.x)
      gs[e] = p.gates[((long long)(t0 + (e >> 1)) * p.heads + c.h) * 2 + (e & 1)];
    copies_commit();
  };
  if (c.first < c.last) fetch(c.first, 0);
  c.load();
  int buffer = 0;
  for (int t0 = c.first; t0 < c.last; t0 += p.chunk, buffer ^= 1) {
    const int count = min(p.chunk, c.last - t0);
    if (t0 + p.chunk < c.last) fetch(t0 + p.chunk, buffer ^ 1);
    else copies_commit();
    copies_wait_all_but_last();
    __syncthreads();
    const float* qs = shared + buffer * per_buffer + c.r * 4;
    const float* ks = qs + p.chunk * kRows;
    const float* vs = shared + buffer * per_buffer + 2 * p.chunk * kRows + c.j;
    const float* gs = shared + buffer * per_buffer + p.chunk * (2 * kRows + p.cols);
    for (int tt = 0; tt < count; ++tt) {
      float k[RP];
      float kd = 0.f, o = 0.f;
#pragma unroll
      for (int i = 0; i < RP; i += 4) {
        const float4 v = *reinterpret_cast<const float4*>(ks + tt * kRows + i * RS);
        k[i] = v.x; k[i + 1] = v.y; k[i + 2] = v.z; k[i + 3] = v.w;
      }
#pragma unroll
      for (int i = 0; i < RP; ++i) kd = fmaf(k[i], c.s[0][i], kd);
#pragma unroll
      for (int d = RS / 2; d > 0; d >>= 1) kd += __shfl_xor_sync(0xffffffffu, kd, d);
      const float fade = gs[2 * tt], beta = gs[2 * tt + 1];
      const float u = beta * (vs[tt * p.cols] - fmaf(fade, kd, kd));
#pragma unroll
      for (int i = 0; i < RP; i += 4) {
        const float4 q = *reinterpret_cast<const float4*>(qs + tt * kRows + i * RS);
#pragma unroll
        for (int n = 0; n < 4; ++n)
          c.s[0][i + n] = fmaf(k[i + n], u, fmaf(fade, c.s[0][i + n], c.s[0][i + n]));
        o = fmaf(c.s[0][i], q.x, o);
        o = fmaf(c.s[0][i + 1], q.y, o);
        o = fmaf(c.s[0][i + 2], q.z, o);
        o = fmaf(c.s[0][i + 3], q.w, o);
      }
#pragma unroll
      for (int d = RS / 2; d > 0; d >>= 1) o += __shfl_xor_sync(0xffffffffu, o, d);
      if (c.live(0) && c.r == 0)
        p.out[((long long)(t0 + tt) * p.heads + c.h) * p.vdim + c.col0 + c.j] = o;
    }
    __syncthreads();
  }
  if (p.keep_state && c.first < c.last) c.store();
}

// Two neighbouring rows. Packed (one 64-bit register, one instruction for both): fewer instructions,
// which pays where a thread has two columns; with one column the longer latency costs more.
template <bool PACKED>
struct Rows2;
template <>
struct Rows2<true> {
  unsigned long long v;
  __device__ __forceinline__ static Rows2 of(float a, float b) {
    Rows2 p;
    asm("mov.b64 %0, {%1, %2};" : "=l"(p.v) : "f"(a), "f"(b));
    return p;
  }
  __device__ __forceinline__ float2 halves() const {
    float2 f;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
    return f;
  }
};
template <>
struct Rows2<false> {
  float x, y;
  __device__ __forceinline__ static Rows2 of(float a, float b) { return {a, b}; }
  __device__ __forceinline__ float2 halves() const { return make_float2(x, y); }
};
__device__ __forceinline__ Rows2<true> fma2(Rows2<true> a, Rows2<true> b, Rows2<true> c) {
  Rows2<true> d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d.v) : "l"(a.v), "l"(b.v), "l"(c.v));
  return d;
}
__device__ __forceinline__ Rows2<false> fma2(Rows2<false> a, Rows2<false> b, Rows2<false> c) {
  return {fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y)};
}
// A running sum of the products of both rows, and what it has come to. (Unpacked it is one chain: two
// were slower, 303 against 254 us for 2,048 tokens of 16 heads of 64 x 64.)
__device__ __forceinline__ Rows2<true> dot2(Rows2<true> a, Rows2<true> b, Rows2<true> sum) {
  return fma2(a, b, sum);
}
__device__ __forceinline__ Rows2<false> dot2(Rows2<false> a, Rows2<false> b, Rows2<false> sum) {
  return {fmaf(a.y, b.y, fmaf(a.x, b.x, sum.x)), 0.f};
}
__device__ __forceinline__ float total(Rows2<true> sum) {
  const float2 f = sum.halves();
  return f.x + f.y;
}
__device__ __forceinline__ float total(Rows2<false> sum) { return sum.x; }

// Four tokens at a time (see above). A thread has one or two columns (CV): what it reads of k and q
// serves them both.
template <int RP, int RS, int CV>
__global__ void __launch_bounds__(256) delta_groups_kernel(const DeltaScan p) {
  static_assert(RS >= 8, "the eight sums of a column end on eight classes of lanes");
  constexpr int kRows = RP * RS;
  constexpr bool kSplit = CV == 2 && RS >= 16;         // the two columns' sums end on different lanes
  using Pair = Rows2<CV == 2>;
  extern __shared__ __align__(16) float shared[];
  let_next_kernel_start();
  wait_for_previous_kernel();
  Columns<RP, RS, CV> c(p);
  const int per_buffer = c.floats(p.chunk / kGroup * kCoef);
  const long long groups0 = first_group(p.cu_seqlens, c.b);
  auto fetch = [&](int t0, int buffer) {
    const int count = min(p.chunk, c.last - t0);
    float* to = shared + buffer * per_buffer;
    c.fetch(to, t0, count, kGroup);
    float* cs = to + p.chunk * (2 * kRows + p.cols);
    const int n = (count + kGroup - 1) / kGroup, g0 = (t0 - c.first) / kGroup;
    for (int e = threadIdx.x; e < n * (kCoef / 4); e += blockDim.x) {
      const int g = e / (kCoef / 4), i = (e - g * (kCoef / 4)) * 4;
      copy16_async(cs + g * kCoef + i, p.coef + ((groups0 + g0 + g) * p.heads + c.h) * kCoef + i);
    }
    copies_commit();
  };
  if (c.first < c.last) fetch(c.first, 0);
  c.load();
  Pair s[CV][RP / 2];
#pragma unroll
  for (int x = 0; x < CV; ++x)
#pragma unroll
    for (int i = 0; i < RP / 2; ++i) s[x][i] = Pair::of(c.s[x][2 * i], c.s[x][2 * i + 1]);
  // after the exchange below a lane holds one of a column's eight sums: with `mine_q` that of query
  // `which`, else that of key `which`; with kSplit that of column `mine_x` only
  const bool mine_q = c.r & (RS / 2), hi = c.r & (RS / 4), lo = c.r & (RS / 8);
  const int which = (hi ? 2 : 0) + (lo ? 1 : 0);
  const int mine_x = kSplit && (c.r & (RS / 16)) ? 1 : 0;
  const bool writes = mine_q && (c.r & ((kSplit ? RS / 16 : RS / 8) - 1)) == 0;
  int buffer = 0;
  for (int t0 = c.first; t0 < c.last; t0 += p.chunk, buffer ^= 1) {
    const int count = min(p.chunk, c.last - t0);
    if (t0 + p.chunk < c.last) fetch(t0 + p.chunk, buffer ^ 1);
    else copies_commit();
    copies_wait_all_but_last();
    __syncthreads();
    const float* qs = shared + buffer * per_buffer + c.r * 4;
    const float* ks = qs + p.chunk * kRows;
    const float* vs = shared + buffer * per_buffer + 2 * p.chunk * kRows + c.j;
    const float* cs = shared + buffer * per_buffer + p.chunk * (2 * kRows + p.cols);
    for (int tt = 0; tt < count; tt += kGroup, cs += kCoef) {
      Pair k[kGroup][RP / 2], kd[CV][kGroup], qd[CV][kGroup];
#pragma unroll
      for (int x = 0; x < CV; ++x)
#pragma unroll
        for (int g = 0; g < kGroup; ++g) kd[x][g] = qd[x][g] = Pair::of(0.f, 0.f);
#pragma unroll
      for (int i = 0; i < RP / 2; i += 2) {
#pragma unroll
        for (int g = 0; g < kGroup; ++g) {
          const float4 a = *reinterpret_cast<const float4*>(ks + (tt + g) * kRows + 2 * i * RS);
          const float4 b = *reinterpret_cast<const float4*>(qs + (tt + g) * kRows + 2 * i * RS);
          k[g][i] = Pair::of(a.x, a.y);
          k[g][i + 1] = Pair::of(a.z, a.w);
#pragma unroll
          for (int x = 0; x < CV; ++x) {
            kd[x][g] = dot2(k[g][i], s[x][i], kd[x][g]);
            kd[x][g] = dot2(k[g][i + 1], s[x][i + 1], kd[x][g]);
            qd[x][g] = dot2(Pair::of(b.x, b.y), s[x][i], qd[x][g]);
            qd[x][g] = dot2(Pair::of(b.z, b.w), s[x][i + 1], qd[x][g]);
          }
        }
      }
      // half of a column's sums to each half of the lanes, then a quarter, then an eighth
      float sum[CV];
#pragma unroll
      for (int x = 0; x < CV; ++x) {
        float four[kGroup];
#pragma unroll
        for (int g = 0; g < kGroup; ++g) {
          const float ka = total(kd[x][g]), qa = total(qd[x][g]);
          four[g] = (mine_q ? qa : ka) + __shfl_xor_sync(0xffffffffu, mine_q ? ka : qa, RS / 2);
        }
        const float two0 = (hi ? four[2] : four[0]) +
                           __shfl_xor_sync(0xffffffffu, hi ? four[0] : four[2], RS / 4);
        const float two1 = (hi ? four[3] : four[1]) +
                           __shfl_xor_sync(0xffffffffu, hi ? four[1] : four[3], RS / 4);
        sum[x] = (lo ? two1 : two0) + __shfl_xor_sync(0xffffffffu, lo ? two0 : two1, RS / 8);
      }
      if constexpr (kSplit) {
        sum[0] = sum[1] = (mine_x ? sum[1] : sum[0]) +
                          __shfl_xor_sync(0xffffffffu, mine_x ? sum[0] : sum[1], RS / 16);
#pragma unroll
        for (int d = RS / 32; d > 0; d >>= 1)
          sum[0] = sum[1] = sum[0] + __shfl_xor_sync(0xffffffffu, sum[0], d);
      } else {
#pragma unroll
        for (int x = 0; x < CV; ++x)
#pragma unroll
          for (int d = RS / 16; d > 0; d >>= 1) sum[x] += __shfl_xor_sync(0xffffffffu, sum[x], d);
      }
      const float4 beta = *reinterpret_cast<const float4*>(cs + kBeta);
      const float4 bc = *reinterpret_cast<const float4*>(cs + kBetaC);
      const float4 end = *reinterpret_cast<const float4*>(cs + kEnd);
      const float4 m0 = *reinterpret_cast<const float4*>(cs + kSolve);
      const float4 m1 = *reinterpret_cast<const float4*>(cs + kSolve + 4);   // (its third: kFade)
      const Pair fade = Pair::of(m1.z, m1.z);
      float u[CV][kGroup];
#pragma unroll
      for (int x = 0; x < CV; ++x) {
        // every lane needs the column's four keys' sums
        const int at = kSplit ? x * (RS / 16) : 0;
        const float k0 = __shfl_sync(0xffffffffu, sum[x], at, RS);
        const float k1 = __shfl_sync(0xffffffffu, sum[x], at + RS / 8, RS);
        const float k2 = __shfl_sync(0xffffffffu, sum[x], at + RS / 4, RS);
        const float k3 = __shfl_sync(0xffffffffu, sum[x], at + RS / 4 + RS / 8, RS);
        const float* v = vs + tt * p.cols + x;
        const float u0 = beta.x * v[0] - bc.x * k0;
        const float u1 = fmaf(-m0.x, u0, beta.y * v[p.cols] - bc.y * k1);
        const float u2 = fmaf(-m0.z, u1, fmaf(-m0.y, u0, beta.z * v[2 * p.cols] - bc.z * k2));
        const float u3 = fmaf(-m1.y, u2, fmaf(-m1.x, u1, fmaf(-m0.w, u0,
                                                              beta.w * v[3 * p.cols] - bc.w * k3)));
        u[x][0] = u0; u[x][1] = u1; u[x][2] = u2; u[x][3] = u3;
      }
      auto move = [&]() {
#pragma unroll
        for (int x = 0; x < CV; ++x) {
          const float e0 = end.x * u[x][0], e1 = end.y * u[x][1], e2 = end.z * u[x][2],
                      e3 = end.w * u[x][3];
          const Pair p0 = Pair::of(e0, e0), p1 = Pair::of(e1, e1), p2 = Pair::of(e2, e2),
                     p3 = Pair::of(e3, e3);
#pragma unroll
          for (int i = 0; i < RP / 2; ++i)
            s[x][i] = fma2(k[3][i], p3, fma2(k[2][i], p2, fma2(k[1][i], p1,
                      fma2(k[0][i], p0, fma2(fade, s[x][i], s[x][i])))));
        }
      };
      // (the state first with two columns, the outputs first with one: each measured against the
      // other, 404 against 427 us and 257 against 312)
      if (CV == 2) move();
      if (writes && tt + which < count) {
        const float4 w = *reinterpret_cast<const float4*>(cs + kOut + 4 * which);
        const float decay = cs[kC + which];
        float* to = p.out + ((long long)(t0 + tt + which) * p.heads + c.h) * p.vdim + c.col0 + c.j;
#pragma unroll
        for (int x = 0; x < CV; ++x) {
          if (kSplit ? x != mine_x || !c.live(x) : !c.live(x)) continue;
          to[x] = fmaf(w.w, u[x][3], fmaf(w.z, u[x][2], fmaf(w.y, u[x][1],
                  fmaf(w.x, u[x][0], decay * sum[x]))));
        }
      }
      if (CV == 1) move();
    }
    __syncthreads();
  }
  if (p.keep_state && c.first < c.last) {
#pragma unroll
    for (int x = 0; x < CV; ++x)
#pragma unroll
      for (int i = 0; i < RP / 2; ++i) {
        const float2 f = s[x][i].halves();
        c.s[x][2 * i] = f.x;
        c.s[x][2 * i + 1] = f.y;
      }
    c.store();
  }
}

template <int RP, int RS>
int launch_scan(DeltaScan p, int sequences, int max_new, bool groups, cudaStream_t stream) {
  constexpr int kRows = RP * RS;
  // two columns a thread where the step's columns then still give every scheduler a warp
  const bool two = groups && p.vdim > 1 &&
                   (long long)p.heads * sequences * p.vdim * RS / 64 >= kTwoWarps * sm_count();
  const int cv = two ? 2 : 1;
  // threads side by side over the columns: blocks of 256 threads, smaller while they do not fill
  // the GPU
  int across = 256 / RS;
  while (across > 4 && across * RS > 64 &&
         (long long)((p.vdim + across * cv - 1) / (across * cv)) * p.heads * sequences < sm_count())
    across /= 2;
  while (across > 4 && across * RS > 64 && across * cv / 2 >= p.vdim) across /= 2;
  const int cols = p.cols = across * cv;
  int chunk = max_new < kChunk ? max_new : kChunk;
  if (groups) chunk = (chunk + kGroup - 1) / kGroup * kGroup;
  auto bytes = [&](int n) {
    return (size_t)2 * (n * (2 * kRows + cols) + (groups ? n / kGroup * kCoef : 2 * n)) * 4;
  };
  constexpr size_t kBudget = 96 * 1024;
  while (chunk > kGroup && bytes(chunk) > kBudget) chunk -= kGroup;
  // (a buffer of gates has an even number of floats: rounded up, the second one stays aligned)
  if (!groups && chunk % 2) ++chunk;
  if (bytes(chunk) > kBudget) return cudaErrorInvalidValue;
  p.chunk = chunk;
  const dim3 grid((unsigned)((p.vdim + cols - 1) / cols), (unsigned)p.heads, (unsigned)sequences);
  auto kernel = two ? delta_groups_kernel<RP, RS, 2>
                    : groups ? delta_groups_kernel<RP, RS, 1> : delta_walk_kernel<RP, RS>;
  const int form = two ? 2 : groups;
  static PerDeviceOnce configured[3];
  if (configured[form].needs()) {
    const cudaError_t e =
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kBudget);
    if (e != cudaSuccess) return (int)e;
    configured[form].done();
  }
  return launch_overlapped(kernel, grid, dim3(across * RS), bytes(chunk), stream, 1, p);
}

template <typename W>
int launch_inputs(const DeltaInputs<W>& p, int sequences, int max_new, cudaStream_t stream) {
  const long long v_width = (long long)p.heads * p.vdim;
  if (max_new == 1 && p.coef == nullptr) {
    const int threads = p.dim <= 64 ? 128 : (2 * p.dim + 31) / 32 * 32;
    const long long units = p.kv_heads + (v_width + threads - 1) / threads;
    if (units > 0x7fffffffLL) return cudaErrorInvalidValue;
    return launch_overlapped(delta_inputs_step_kernel<W>, dim3((unsigned)units, (unsigned)sequences),
                             dim3(threads), (size_t)2 * p.dim * sizeof(float), stream, 1, p);
  }
#define SAKV_INPUTS(PER, TAPS)                                                                   \
  do {                                                                                           \
    const long long units = p.kv_heads + (v_width + 32 * PER - 1) / (32 * PER);                  \
    const long long warps = units * ((max_new + kGroup - 1) / kGroup);                           \
    const long long blocks = (warps + 3) / 4;                                                    \
    if (blocks > 0x7fffffffLL) return cudaErrorInvalidValue;                                     \
    return launch_overlapped(delta_inputs_kernel<PER, TAPS, W>,                                  \
                             dim3((unsigned)blocks, (unsigned)sequences), dim3(128), 0, stream,  \
                             1, p);                                                              \
  } while (0)
  if (p.taps == 4) {                                   // (the usual width of these convolutions)
    if (p.dim <= 32) SAKV_INPUTS(1, 4);
    if (p.dim <= 64) SAKV_INPUTS(2, 4);
    if (p.dim <= 128) SAKV_INPUTS(4, 4);
    if (p.dim <= 256) SAKV_INPUTS(8, 4);
  }
  if (p.dim <= 32) SAKV_INPUTS(1, 0);
  if (p.dim <= 64) SAKV_INPUTS(2, 0);
  if (p.dim <= 128) SAKV_INPUTS(4, 0);
  if (p.dim <= 256) SAKV_INPUTS(8, 0);
  SAKV_INPUTS(16, 0);
#undef SAKV_INPUTS
}

}  // namespace

SAKV_EXPORT int sakv_delta_coefficients() { return kCoef; }

// proj: fp32 [tokens, stride] with the pre-activations of q (kv_heads * dim), k (the same), v
// (heads * vdim) in its first columns, the decays' at a_off and the betas' at b_off (heads each).
// conv: [channels, taps] of `w_dtype`, channels = 2 kv_heads dim + heads vdim; a (-exp(A_log)),
// dt_bias: fp32 [heads]. conv_state: fp32 [slots, taps - 1, channels], read; with move_state (a
// step in which every sequence brings one token) also moved up by the token's inputs. prepared:
// fp32 [tokens, channels] = unit q times q_scale, unit k, v; gates: fp32 [tokens, heads, 2] =
// (decay less one, beta); coef (null: not made): fp32 [tokens / 4 + sequences, heads,
// sakv_delta_coefficients()]. max_new: the most tokens a sequence brings.
SAKV_EXPORT int sakv_delta_inputs(const float* proj, long long stride, int a_off, int b_off,
                                  const void* conv, int w_dtype, const float* a,
                                  const float* dt_bias, float* conv_state,
                                  const int32_t* cu_seqlens, const int32_t* slots, float* prepared,
                                  float* gates, float* coef, int sequences, int max_new, int heads,
                                  int kv_heads, int dim, int vdim, int taps, int move_state,
                                  float q_scale, float unit_eps, cudaStream_t stream) {
  if (sequences < 0 || sequences > 65535 || max_new < 0 || heads <= 0 || kv_heads <= 0 ||
      heads % kv_heads || dim <= 0 || dim > 512 || vdim <= 0 || taps < 1 || taps > 64 ||
      (move_state && max_new > 1))
    return cudaErrorInvalidValue;
  if (sequences == 0 || max_new == 0) return 0;
  const int channels = 2 * kv_heads * dim + heads * vdim;
#define SAKV_IN(W)                                                                               \
  return launch_inputs(DeltaInputs<W>{proj, stride, a_off, b_off, (const W*)conv, a, dt_bias,    \
                                      conv_state, cu_seqlens, slots, prepared, gates, coef,      \
                                      heads, kv_heads, dim, vdim, taps, channels, move_state,    \
                                      q_scale, unit_eps},                                        \
                       sequences, max_new, stream)
  if (w_dtype == SAKV_F32) SAKV_IN(float);
  if (w_dtype == SAKV_BF16) SAKV_IN(__nv_bfloat16);
#undef SAKV_IN
  return cudaErrorInvalidValue;
}

// prepared, gates, coef: from `sakv_delta_inputs` (16-byte aligned). state: fp32 [slots, heads,
// vdim, dim], read and (with keep_state) left. out: fp32 [tokens, heads * vdim]. coef null: one
// token at a time; else four.
SAKV_EXPORT int sakv_delta_scan(const float* prepared, const float* gates, const float* coef,
                                float* state, const int32_t* cu_seqlens, const int32_t* slots,
                                float* out, int sequences, int max_new, int heads, int kv_heads,
                                int dim, int vdim, int keep_state, cudaStream_t stream) {
  if (sequences < 0 || sequences > 65535 || max_new < 0 || heads <= 0 || heads > 65535 ||
      kv_heads <= 0 || heads % kv_heads || dim <= 0 || dim > 512 || vdim <= 0 ||
      (((uintptr_t)prepared | (uintptr_t)coef | (uintptr_t)state) & 15))
    return cudaErrorInvalidValue;
  if (sequences == 0 || max_new == 0) return 0;
  const int channels = 2 * kv_heads * dim + heads * vdim;
  const DeltaScan p = {prepared, gates, coef,     state, cu_seqlens, slots, out,       heads,
                       kv_heads, dim,   vdim, channels, 0,          0,     keep_state};
  const bool groups = coef != nullptr;
  if (dim <= 32) return launch_scan<4, 8>(p, sequences, max_new, groups, stream);
  if (dim <= 64) return launch_scan<8, 8>(p, sequences, max_new, groups, stream);
  if (dim <= 128) return launch_scan<8, 16>(p, sequences, max_new, groups, stream);
  if (dim <= 256) return launch_scan<8, 32>(p, sequences, max_new, groups, stream);
  return launch_scan<16, 32>(p, sequences, max_new, groups, stream);
}
