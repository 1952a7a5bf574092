// The recurrence of a gated delta rule: per request and head a state S [dim, vdim] in 32-bit floats that
// is carried from token to token.  With unit vectors k and q (q also times dim^-1/2), a decay g and a step
// size beta per head and token:
//
//   S_t = g_t S_{t-1} + k_t u_t^T   with   u_t = beta_t (v_t - g_t S_{t-1}^T k_t);     o_t = S_t^T q_t
//   g = exp(-exp(A_log) softplus(a + dt_bias)),  beta = sigmoid(b)
//
// The columns of S are independent of each other given u, so a thread group of SL lanes owns a few columns
// and splits the key channels among its lanes.
//
// Several tokens are taken at once (TB = 4 in long segments).  Within such a block the state before it, S0,
// enters every token's reads linearly: with G_t = g_1 .. g_t,
//
//   u_t = beta_t (v_t - G_t S0^T k_t - sum_{s<t} (G_t / G_s) (k_s . k_t) u_s)
//   o_t = G_t S0^T q_t + sum_{s<=t} (G_t / G_s) (k_s . q_t) u_s
//   S   = G_T S0 + sum_s (G_T / G_s) k_s u_s^T
//
// so the block's eight dot products with S0 are summed over the lanes together, one latency for four tokens.
// G_t / G_s is always taken as the product g_{s+1} .. g_t: nothing divides, decays may be zero.
// delta_prepare_kernel leaves, per token and head, the twelve numbers these lines need (the inverse norms of
// k and q are part of them, so the rows themselves are used as they are):
//   [G_t |k_t|^-1, G_t |q_t|^-1 c, beta_t, (G_T / G_t) |k_t|^-1 | (G_t / G_s) k_s . k_t for s < t, G_T |
//    (G_t / G_s) k_s . q_t for s <= t]
//
// Blocks start at the segment's first row of the step, so where a block's border lies depends on how a
// prompt was cut; that changes the order of additions only.
#include "common.cuh"
#include "copy_async.cuh"
#include "lane_sums.cuh"

namespace mlr {

constexpr int DELTA_COEF = 12;

struct DeltaArgs {
  const float *q, *k, *v, *a, *b;       // row-major views, one row per token
  long long q_stride, k_stride, v_stride, a_stride, b_stride;
  const float *dt_bias, *A_log;         // [heads]
  float* coef;                          // [rows, heads, 12] (TB > 1)
  float* states;                        // [slots, heads, vdim, dim]
  float* y;                             // [rows, heads * vdim]
  const int *seg_q_start, *seg_q_len, *seg_slot;
  int heads, kv_heads, dim, vdim;
  float unit_eps, q_scale;
};

__device__ __forceinline__ float delta_decay(float raw, float bias, float a_log) {
  const float z = raw + bias;
  const float dt = z > 20.f ? z : log1pf(expf(z));
  return expf(-expf(a_log) * dt);
}
__device__ __forceinline__ float delta_beta(float raw) { return 1.f / (1.f + expf(-raw)); }

// One warp per block of four tokens and key/value head: the block's products of keys and queries, then
// the numbers above for every head that reads this key/value head (one lane per head).
// grid: (token block groups, segments, kv heads)
constexpr int PREP_WARPS = 4;
__global__ void __launch_bounds__(PREP_WARPS * 32)
delta_prepare_kernel(DeltaArgs p) {
  // The recurrence behind this kernel is few blocks that run long: brought in while this kernel's many blocks
  // still fill the SMs, they would land several to an SM.  So there is no early trigger here.
  pdl_wait();
  const int seg = blockIdx.y, kv = blockIdx.z;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int q_len = p.seg_q_len[seg];
  const int t0 = (blockIdx.x * PREP_WARPS + warp) * 4;
  if (t0 >= q_len) return;
  const size_t row0 = (size_t)p.seg_q_start[seg] + t0;
  const int count = min(4, q_len - t0);
  float kk[4][4], qk[4][4], qq[4];      // kk[t][s] for s <= t, qk[t][s] = q_t . k_s for s <= t
#pragma unroll
  for (int t = 0; t < 4; ++t) {
    qq[t] = 0.f;
#pragma unroll
    for (int s = 0; s < 4; ++s) kk[t][s] = qk[t][s] = 0.f;
  }
  for (int d = lane; d < p.dim; d += 32) {
    float kv_[4], qv[4];
#pragma unroll
    for (int t = 0; t < 4; ++t) {
      kv_[t] = t < count ? __ldcg(p.k + (row0 + t) * p.k_stride + (size_t)kv * p.dim + d) : 0.f;
      qv[t] = t < count ? __ldcg(p.q + (row0 + t) * p.q_stride + (size_t)kv * p.dim + d) : 0.f;
    }
#pragma unroll
    for (int t = 0; t < 4; ++t) {
      qq[t] = fmaf(qv[t], qv[t], qq[t]);
#pragma unroll
      for (int s = 0; s <= t; ++s) {
        kk[t][s] = fmaf(kv_[t], kv_[s], kk[t][s]);
        qk[t][s] = fmaf(qv[t], kv_[s], qk[t][s]);
      }
    }
  }
#pragma unroll
  for (int t = 0; t < 4; ++t) {
    qq[t] = warp_sum(qq[t]);
#pragma unroll
    for (int s = 0; s <= t; ++s) {
      kk[t][s] = warp_sum(kk[t][s]);
      qk[t][s] = warp_sum(qk[t][s]);
    }
  }
  float rk[4], rq[4];
#pragma unroll
  for (int t = 0; t < 4; ++t) {
    rk[t] = 1.f / sqrtf(kk[t][t] + p.unit_eps);
    rq[t] = p.q_scale / sqrtf(qq[t] + p.unit_eps);
  }
  const int per = p.heads / p.kv_heads;
  for (int i = lane; i < per; i += 32) {
    const int head = kv * per + i;
    float g[4], beta[4];
#pragma unroll
    for (int t = 0; t < 4; ++t) {
      g[t] = 1.f;
      beta[t] = 0.f;
      if (t < count) {
        g[t] = delta_decay(__ldcg(p.a + (row0 + t) * p.a_stride + head), p.dt_bias[head], p.A_log[head]);
        beta[t] = delta_beta(__ldcg(p.b + (row0 + t) * p.b_stride + head));
      }
    }
    const float all = g[0] * g[1] * g[2] * g[3];
    float before = 1.f, behind = all;
#pragma unroll
    for (int t = 0; t < 4; ++t) {
      before *= g[t];
      behind = 1.f;
#pragma unroll
      for (int s = t + 1; s < 4; ++s) behind *= g[s];
      if (t >= count) continue;
      float l[3] = {0.f, 0.f, 0.f}, m[4] = {0.f, 0.f, 0.f, 0.f};
      float between = 1.f;
#pragma unroll
      for (int s = t; s >= 0; --s) {      // between = g[s + 1] .. g[t]
        m[s] = between * rk[s] * rq[t] * qk[t][s];
        if (s < t) l[s < 3 ? s : 0] = between * rk[s] * rk[t] * kk[t][s];
        between *= g[s];
      }
      float4* dst = reinterpret_cast<float4*>(p.coef + ((row0 + t) * p.heads + head) * DELTA_COEF);
      dst[0] = make_float4(before * rk[t], before * rq[t], beta[t], behind * rk[t]);
      dst[1] = make_float4(l[0], l[1], l[2], all);
      dst[2] = make_float4(m[0], m[1], m[2], m[3]);
    }
  }
}

// grid: (segments, heads, column blocks).  A group of SL lanes holds C columns of the head's state, each
// lane E key channels of them (in interleaved pieces of four: neighbouring lanes read neighbouring 16-byte
// pieces of a staged row).  TB tokens per turn; TB == 1 computes its numbers itself.  WIDE: rows are staged
// in 16-byte pieces (sizes and strides multiples of four floats, pointers aligned).
template <int E, int SL, int C, int TB, bool WIDE, int THREADS>
__global__ void __launch_bounds__(THREADS)
delta_scan_kernel(DeltaArgs p) {
  pdl_trigger();
  extern __shared__ __align__(16) float shared[];
  constexpr int GROUPS = THREADS / SL, COLS = GROUPS * C;
  constexpr int N = TB * C;
  constexpr int TOKENS = SL == 32 ? 16 : 32;      // tokens staged at once
  const int D = p.dim, V = p.vdim;
  constexpr int pitch = E * SL;                                       // staged rows of keys and queries, filled up with zeros
  const int buffer = TOKENS * (2 * pitch + COLS + DELTA_COEF);  // floats of one staging buffer
  const int seg = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * COLS;
  const int kv = head / (p.heads / p.kv_heads);
  const int lane = threadIdx.x & 31, s = threadIdx.x % SL, group = threadIdx.x / SL;
  const float a_log = p.A_log[head], bias = p.dt_bias[head];
  pdl_wait();
  const int q_start = p.seg_q_start[seg], q_len = p.seg_q_len[seg];

  // zeros that no copy overwrites: behind the rows' D entries
  if (D < pitch) {
    for (int idx = threadIdx.x; idx < 4 * TOKENS * (pitch - D); idx += THREADS) {
      const int row = idx / (pitch - D), d = D + idx - row * (pitch - D);
      shared[(row / (2 * TOKENS)) * buffer + (row % (2 * TOKENS)) * pitch + d] = 0.f;
    }
  }
  auto stage = [&](int t0, int which) {
    float* k_rows = shared + which * buffer;
    float* q_rows = k_rows + TOKENS * pitch;
    float* v_rows = q_rows + TOKENS * pitch;
    float* coef = v_rows + TOKENS * COLS;
    const int tokens = min(TOKENS, q_len - t0);
    const size_t row0 = (size_t)(q_start + t0);
    if (WIDE) {
      const int per_row = D >> 2;
      for (int idx = threadIdx.x; idx < tokens * per_row; idx += THREADS) {
        const int t = idx / per_row, d = (idx - t * per_row) << 2;
        copy_async_16(k_rows + t * pitch + d, p.k + (row0 + t) * p.k_stride + (size_t)kv * D + d);
        copy_async_16(q_rows + t * pitch + d, p.q + (row0 + t) * p.q_stride + (size_t)kv * D + d);
      }
      constexpr int PIECES = COLS / 4;
      for (int idx = threadIdx.x; idx < tokens * PIECES; idx += THREADS) {
        const int t = idx / PIECES, c = (idx - t * PIECES) << 2;
        if (col0 + c < V) copy_async_16(v_rows + t * COLS + c, p.v + (row0 + t) * p.v_stride + (size_t)head * V + col0 + c);
      }
    } else {
      for (int idx = threadIdx.x; idx < tokens * D; idx += THREADS) {
        const int t = idx / D, d = idx - t * D;
        copy_async_4(k_rows + t * pitch + d, p.k + (row0 + t) * p.k_stride + (size_t)kv * D + d);
        copy_async_4(q_rows + t * pitch + d, p.q + (row0 + t) * p.q_stride + (size_t)kv * D + d);
      }
      for (int idx = threadIdx.x; idx < tokens * COLS; idx += THREADS) {
        const int t = idx / COLS, c = idx - t * COLS;
        if (col0 + c < V) copy_async_4(v_rows + idx, p.v + (row0 + t) * p.v_stride + (size_t)head * V + col0 + c);
      }
    }
    if (TB > 1) {
      for (int idx = threadIdx.x; idx < tokens * 3; idx += THREADS) {
        const int t = idx / 3, c = (idx - t * 3) << 2;
        copy_async_16(coef + t * DELTA_COEF + c, p.coef + ((row0 + t) * p.heads + head) * DELTA_COEF + c);
      }
    } else if (threadIdx.x < tokens) {
      copy_async_4(coef + threadIdx.x * DELTA_COEF, p.a + (row0 + threadIdx.x) * p.a_stride + head);
      copy_async_4(coef + threadIdx.x * DELTA_COEF + 1, p.b + (row0 + threadIdx.x) * p.b_stride + head);
    }
    copy_async_commit();
    if (TB > 1 && tokens % TB != 0) {      // the rest of the last block of tokens: nothing is read, written or forgotten
      const int fill = TB - tokens % TB;
      for (int idx = threadIdx.x; idx < fill * pitch; idx += THREADS) {
        k_rows[tokens * pitch + idx] = 0.f;
        q_rows[tokens * pitch + idx] = 0.f;
      }
      for (int idx = threadIdx.x; idx < fill * COLS; idx += THREADS) v_rows[tokens * COLS + idx] = 0.f;
      for (int idx = threadIdx.x; idx < fill * DELTA_COEF; idx += THREADS) coef[tokens * DELTA_COEF + idx] = 0.f;
    }
  };

  stage(0, 0);
  float* state = p.states + ((size_t)p.seg_slot[seg] * p.heads + head) * V * D;
  auto entry = [&](int i) { return (((i >> 2) * SL + s) << 2) + (i & 3); };      // key channel of a lane's i-th number
  int column[C];
#pragma unroll
  for (int c = 0; c < C; ++c) column[c] = col0 + group * C + c;
  float S[C][E];
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const bool mine = column[c] < V;
    const float* src = state + (size_t)(mine ? column[c] : 0) * D;
    if (WIDE) {
#pragma unroll
      for (int i = 0; i < E; i += 4) {
        float4 v4 = make_float4(0.f, 0.f, 0.f, 0.f);
        if (mine && entry(i) < D) v4 = __ldcg(reinterpret_cast<const float4*>(src + entry(i)));
        S[c][i] = v4.x; S[c][i + 1] = v4.y; S[c][i + 2] = v4.z; S[c][i + 3] = v4.w;
      }
    } else {
#pragma unroll
      for (int i = 0; i < E; ++i) S[c][i] = mine && entry(i) < D ? __ldcg(src + entry(i)) : 0.f;
    }
  }

  int which = 0;
  for (int t0 = 0; t0 < q_len; t0 += TOKENS, which ^= 1) {
    const int tokens = min(TOKENS, q_len - t0);
    const bool more = t0 + TOKENS < q_len;
    if (more) stage(t0 + TOKENS, which ^ 1);
    if (more) copy_async_wait<1>(); else copy_async_wait<0>();
    __syncthreads();
    const float* k_rows = shared + which * buffer;
    const float* q_rows = k_rows + TOKENS * pitch;
    const float* v_rows = q_rows + TOKENS * pitch;
    float* coef = const_cast<float*>(v_rows) + TOKENS * COLS;
    if (TB == 1) {
      for (int t = threadIdx.x >> 5; t < tokens; t += THREADS / 32) {
        float kk = 0.f, qq = 0.f, qk = 0.f;
        for (int d = lane; d < D; d += 32) {
          const float kd = k_rows[t * pitch + d], qd = q_rows[t * pitch + d];
          kk = fmaf(kd, kd, kk);
          qq = fmaf(qd, qd, qq);
          qk = fmaf(qd, kd, qk);
        }
        kk = warp_sum(kk);
        qq = warp_sum(qq);
        qk = warp_sum(qk);
        if (lane == 0) {
          float* c = coef + t * DELTA_COEF;
          const float g = delta_decay(c[0], bias, a_log), beta = delta_beta(c[1]);
          const float rk = 1.f / sqrtf(kk + p.unit_eps), rq = p.q_scale / sqrtf(qq + p.unit_eps);
          c[0] = g * rk;
          c[1] = g * rq;
          c[2] = beta;
          c[3] = rk;
          c[7] = g;
          c[8] = rk * rq * qk;
        }
      }
      __syncthreads();
    }
    // a block's rows are read from shared memory while the block before is worked on
    float4 k_next[TB][E / 4], q_next[TB][E / 4];
    auto read_rows = [&](int t) {
#pragma unroll
      for (int n = 0; n < TB; ++n)
#pragma unroll
        for (int i = 0; i < E / 4; ++i) {
          k_next[n][i] = *reinterpret_cast<const float4*>(k_rows + (t + n) * pitch + entry(4 * i));
          q_next[n][i] = *reinterpret_cast<const float4*>(q_rows + (t + n) * pitch + entry(4 * i));
        }
    };
    constexpr bool AHEAD = E == 4;      // with more key channels per lane the registers do better otherwise
    if (AHEAD) read_rows(0);
    for (int t = 0; t < tokens; t += TB) {
      // the block's dot products with the state before it; the keys stay in registers for the update
      if (!AHEAD) read_rows(t);
      float kd[TB][E], dk[N], dq[N];
#pragma unroll
      for (int n = 0; n < N; ++n) dk[n] = dq[n] = 0.f;
#pragma unroll
      for (int n = 0; n < TB; ++n) {
#pragma unroll
        for (int i = 0; i < E / 4; ++i) {
          kd[n][4 * i] = k_next[n][i].x; kd[n][4 * i + 1] = k_next[n][i].y;
          kd[n][4 * i + 2] = k_next[n][i].z; kd[n][4 * i + 3] = k_next[n][i].w;
        }
      }
#pragma unroll
      for (int i = 0; i < E / 4; ++i) {
#pragma unroll
        for (int n = 0; n < TB; ++n) {
          const float qd[4] = {q_next[n][i].x, q_next[n][i].y, q_next[n][i].z, q_next[n][i].w};
#pragma unroll
          for (int c = 0; c < C; ++c) {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              dk[n * C + c] = fmaf(kd[n][4 * i + j], S[c][4 * i + j], dk[n * C + c]);
              dq[n * C + c] = fmaf(qd[j], S[c][4 * i + j], dq[n * C + c]);
            }
          }
        }
      }
      if (AHEAD && t + TB < tokens) read_rows(t + TB);
      // the key sums are needed by every lane of the group (the u follow from them), the query sums by one
      if (N <= SL) {
        spread_sums<N, SL>(dk, lane);
        const float mine = dk[0];
#pragma unroll
        for (int n = 0; n < N; ++n) dk[n] = __shfl_sync(0xffffffffu, mine, n * (SL / N), SL);
      } else {
#pragma unroll
        for (int m = SL / 2; m > 0; m >>= 1)
#pragma unroll
          for (int n = 0; n < N; ++n) dk[n] += __shfl_xor_sync(0xffffffffu, dk[n], m);
      }
      const int first = spread_sums<N, SL>(dq, lane);
      float u[TB][C], w[TB], all = 1.f;
#pragma unroll
      for (int n = 0; n < TB; ++n) {
        const float4 c0 = *reinterpret_cast<const float4*>(coef + (t + n) * DELTA_COEF);
        const float4 c1 = *reinterpret_cast<const float4*>(coef + (t + n) * DELTA_COEF + 4);
        w[n] = c0.w;
        if (n == 0) all = c1.w;
        const float l[3] = {c1.x, c1.y, c1.z};
#pragma unroll
        for (int c = 0; c < C; ++c) {
          float read = c0.x * dk[n * C + c];
#pragma unroll
          for (int m = 0; m < n; ++m) read = fmaf(l[m < 3 ? m : 0], u[m][c], read);
          u[n][c] = c0.z * (v_rows[(t + n) * COLS + group * C + c] - read);
        }
      }
      // this lane's outputs: number `first + i` is token number / C, column number % C
      constexpr int HELD = N > SL ? N / SL : 1;
      if (N >= SL || (s & (SL / N - 1)) == 0) {
#pragma unroll
        for (int i = 0; i < HELD; ++i) {
          const int number = first + i, n = number / C, c = number % C;
          if (t + n < tokens && col0 + group * C + c < V) {
            const float b = coef[(t + n) * DELTA_COEF + 1];
            const float4 m4 = *reinterpret_cast<const float4*>(coef + (t + n) * DELTA_COEF + 8);      // zero beyond the token
            const float m[4] = {m4.x, m4.y, m4.z, m4.w};
            float o = b * dq[i];
#pragma unroll
            for (int e = 0; e < TB; ++e) {
              float ue = u[e][0];
#pragma unroll
              for (int cc = 1; cc < C; ++cc) ue = c == cc ? u[e][cc] : ue;
              o = fmaf(m[e], ue, o);
            }
            p.y[((size_t)(q_start + t0 + t + n) * p.heads + head) * V + col0 + group * C + c] = o;
          }
        }
      }
#pragma unroll
      for (int n = 0; n < TB; ++n)
#pragma unroll
        for (int c = 0; c < C; ++c) u[n][c] *= w[n];
#pragma unroll
      for (int c = 0; c < C; ++c) {
#pragma unroll
        for (int i = 0; i < E; ++i) {
          float next = all * S[c][i];
#pragma unroll
          for (int n = 0; n < TB; ++n) next = fmaf(kd[n][i], u[n][c], next);
          S[c][i] = next;
        }
      }
    }
    __syncthreads();      // the next turn of the loop stages into this buffer
  }
#pragma unroll
  for (int c = 0; c < C; ++c) {
    if (column[c] >= V) continue;
    float* dst = state + (size_t)column[c] * D;
    if (WIDE) {
#pragma unroll
      for (int i = 0; i < E; i += 4)
        if (entry(i) < D) *reinterpret_cast<float4*>(dst + entry(i)) = make_float4(S[c][i], S[c][i + 1], S[c][i + 2], S[c][i + 3]);
    } else {
#pragma unroll
      for (int i = 0; i < E; ++i)
        if (entry(i) < D) dst[entry(i)] = S[c][i];
    }
  }
}

template <int E, int SL, int C, int TB, bool WIDE, int THREADS = 128>
static int launch_delta(const DeltaArgs& p, int segments, cudaStream_t stream) {
  constexpr int COLS = THREADS / SL * C;
  constexpr int pitch = E * SL;
  constexpr int TOKENS = SL == 32 ? 16 : 32;
  const size_t shared = sizeof(float) * 2 * (size_t)TOKENS * (2 * pitch + COLS + DELTA_COEF);
  if (shared > 227 * 1024) return MLR_TOO_LARGE;
  auto kernel = delta_scan_kernel<E, SL, C, TB, WIDE, THREADS>;
  if (shared > 48 * 1024) {
    cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared);
    if (err != cudaSuccess) return (int)err;
  }
  launch_kernel(kernel, dim3(segments, p.heads, (p.vdim + COLS - 1) / COLS), dim3(THREADS), shared, stream, p);
  return launch_status();
}

}  // namespace mlr

using namespace mlr;

MLR_DEFINE_PDL_SWITCH

// q, k: float32 rows of kv_heads * dim entries; v: rows of heads * vdim entries; a, b: rows of `heads` entries
// (each with its own row stride); dt_bias, A_log: float32 [heads]; coef: float32 scratch [rows, heads, 12], or
// null (then tokens are taken one by one); states: float32 [slots, heads, vdim, dim] (the transposed S);
// y: float32 [rows, heads * vdim].  max_q_len: the longest segment of the step.
MLR_EXPORT int mlr_delta_rule_scan(const float* q, long long q_stride, const float* k, long long k_stride, const float* v,
                                   long long v_stride, const float* a, long long a_stride, const float* b, long long b_stride,
                                   const float* dt_bias, const float* A_log, float* coef, float* states, float* y,
                                   const int* seg_q_start, const int* seg_q_len, const int* seg_slot, int segments,
                                   int max_q_len, int heads, int kv_heads, int dim, int vdim, float unit_eps, float q_scale,
                                   cudaStream_t stream) {
  if (segments == 0) return MLR_OK;
  if (segments < 0 || max_q_len <= 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || dim <= 0 || vdim <= 0)
    return MLR_BAD_SIZE;
  if (dim > 512 || heads > 65535 || segments > 65535 || vdim > 65535) return MLR_TOO_LARGE;
  DeltaArgs p{q, k, v, a, b, q_stride, k_stride, v_stride, a_stride, b_stride, dt_bias, A_log, coef, states, y,
              seg_q_start, seg_q_len, seg_slot, heads, kv_heads, dim, vdim, unit_eps, q_scale};
  auto multiple = [](long long n) { return n % 4 == 0; };
  auto aligned = [](const void* ptr) { return (reinterpret_cast<uintptr_t>(ptr) & 15) == 0; };
  const bool wide = multiple(dim) && multiple(vdim) && multiple(q_stride) && multiple(k_stride) && multiple(v_stride) &&
                    aligned(q) && aligned(k) && aligned(v) && aligned(states) && aligned(coef);
  if (wide && coef != nullptr && max_q_len > 1) {
    const int blocks = (max_q_len + 4 * PREP_WARPS - 1) / (4 * PREP_WARPS);
    launch_kernel(delta_prepare_kernel, dim3(blocks, segments, kv_heads), dim3(PREP_WARPS * 32), 0, stream, p);
    const int status = launch_status();
    if (status != MLR_OK) return status;
    if (dim <= 32) return launch_delta<4, 8, 1, 4, true>(p, segments, stream);
    if (dim <= 64) return launch_delta<4, 16, 1, 4, true>(p, segments, stream);
    if (dim <= 128) {
      // one column per group while that many warps still fit the device well, else two (a row read from shared
      // memory then serves both): 2,048 tokens, 32 heads of 128 x 64: 335 / 398 us, of 128 x 128: 521 / 420 us
      if ((long long)segments * heads * vdim <= 20LL * sm_count()) return launch_delta<8, 16, 1, 4, true, 256>(p, segments, stream);
      return launch_delta<8, 16, 2, 4, true>(p, segments, stream);
    }
    if (dim <= 256) return launch_delta<8, 32, 2, 4, true>(p, segments, stream);
    return launch_delta<16, 32, 2, 4, true>(p, segments, stream);
  }
  if (wide) {
    if (dim <= 32) return launch_delta<4, 8, 1, 1, true>(p, segments, stream);
    if (dim <= 64) return launch_delta<8, 8, 1, 1, true>(p, segments, stream);
    if (dim <= 128) return launch_delta<16, 8, 1, 1, true>(p, segments, stream);
    if (dim <= 256) return launch_delta<16, 16, 1, 1, true>(p, segments, stream);
    return launch_delta<16, 32, 1, 1, true>(p, segments, stream);
  }
  if (dim <= 32) return launch_delta<4, 8, 1, 1, false>(p, segments, stream);
  if (dim <= 128) return launch_delta<16, 8, 1, 1, false>(p, segments, stream);
  return launch_delta<16, 32, 1, 1, false>(p, segments, stream);
}
