// A matrix memory with exponential gates (the mLSTM of xLSTM): per request and head a memory S [dim, vdim] and a
// normaliser n [dim] in 32-bit floats that are carried from token to token,
//
//   i = cap tanh((i_raw + i_bias) / cap),   f = logsigmoid(cap tanh((f_raw + f_bias) / cap))       (logarithms)
//   m_t = max(f + m_{t-1}, i)
//   S_t = e^(f + m_{t-1} - m_t) S_{t-1} + e^(i - m_t) k_t v_t^T,      n_t likewise with k_t alone
//   o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + guard),           q = q_raw * dim^-1/2
//   out = o / rms(o) * weight * sigmoid(gate)                          (rms over a head's channels)
//
// The state is kept transposed with n as one more value channel (whose value is 1): [vdim + 1, dim].
//
// matrix_memory_decode_kernel   steps of single rows: everything above in one launch, a block per (request, head).
// matrix_memory_gates_kernel    per token and head [keep, write, e^(-m)]: the running maximum is an associative scan of
//                               maps m -> max(a + m, b).  Wherever m appears the same rounded m_t is used, so what m's
//                               own rounding does to S cancels out.
// matrix_memory_scan_kernel     the recurrence of longer segments, token after token, value channels over blocks.
// matrix_memory_finish_kernel   normaliser, head norm, weight and gate of the scan's rows.
//
// In bfloat16, prompts take chunks of 64 tokens through the tensor cores instead of the token-by-token scan.  q, k and
// v are projections and enter rounded to bfloat16; everything else stays 32-bit: products of a 32-bit operand are
// taken of its three bfloat16 parts (24 bits), sums are 32-bit.  With K_t the product of the keeps of a chunk's tokens up to
// t and D_ts = write_s times the keeps of s + 1 .. t (products of numbers up to one, no differences of logarithms),
//
//   S^T q_t (of token t) = K_t S_before^T q_t + sum_{s <= t} A_ts v_s    with  A_ts = D_ts (k_s . q_t)
//   S_behind = K_last S_before + sum_s k_s (D_last,s v_s)^T
//
// matrix_memory_pairs_kernel    all chunks at once: A, D_last and K of every chunk, q, k and v as bfloat16.
// matrix_memory_chunks_kernel   the chunks of a (request, head) one after the other, value channels over blocks; the
//                               state stays in registers as accumulators.
#include "mma_attention.cuh"
#include "copy_async.cuh"
#include "lane_sums.cuh"

namespace mlr {

struct MemoryArgs {
  const float *q, *k, *v, *i_raw, *f_raw, *gate;      // row-major views, one row per token
  long long q_stride, k_stride, v_stride, i_stride, f_stride, gate_stride;
  const float *i_bias, *f_bias;         // [heads]
  const float* weight;                  // [heads * vdim]
  float4* coef;                         // [rows, heads]: keep, write, e^(-m), unused
  float* reads;                         // [rows, heads, vdim]: S^T q before the normaliser
  float* norms;                         // [rows, heads]: n . q
  float* pairs;                         // chunks: [rows, heads, 64], A
  float2* factors;                      // chunks: [rows, heads]: D_last and K
  bf16 *q16, *k16, *v16;                // chunks: [rows, heads * dim], the same, [rows, heads * vdim]
  float* states;                        // [slots, heads, vdim + 1, dim]
  float* maxima;                        // [slots, heads]
  const int *seg_q_start, *seg_q_len, *seg_slot;
  int heads, dim, vdim;
  float cap, guard, eps, q_scale;
};

__device__ __forceinline__ float capped(float raw, float cap) { return cap * tanhf(raw / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// ------------------------------------------------------------------ single rows
constexpr int DECODE_THREADS = 256;
constexpr int DECODE_WARPS = DECODE_THREADS / 32;

// PIECES: 16-byte pieces of a state row per lane (dim <= 128 * PIECES, rows and pointers aligned), or 0: any
// size, number by number.  grid: (segments, heads).
template <typename T, int PIECES>
__global__ void __launch_bounds__(DECODE_THREADS)
matrix_memory_decode_kernel(MemoryArgs p, T* __restrict__ out) {
  pdl_trigger();
  extern __shared__ __align__(16) float shared[];      // [vdim + 1] reads
  __shared__ float scratch[32];
  const int seg = blockIdx.x, head = blockIdx.y, D = p.dim, V = p.vdim;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const size_t slot_head = (size_t)p.seg_slot[seg] * p.heads + head;
  const size_t row = p.seg_q_start[seg];
  float* state = p.states + slot_head * (size_t)(V + 1) * D;
  const float i_bias = p.i_bias[head], f_bias = p.f_bias[head];
  pdl_wait();
  const float i_raw = __ldcg(p.i_raw + row * p.i_stride + head), f_raw = __ldcg(p.f_raw + row * p.f_stride + head);
  const float m_old = __ldcg(p.maxima + slot_head);
  const float* q = p.q + row * p.q_stride + (size_t)head * D;
  const float* k = p.k + row * p.k_stride + (size_t)head * D;
  const float* v = p.v + row * p.v_stride + (size_t)head * V;
  float m_new = 0.f, keep = 0.f, write = 0.f;
  auto gates = [&]() {
    const float log_in = capped(i_raw + i_bias, p.cap), log_forget = log_sigmoid(capped(f_raw + f_bias, p.cap));
    m_new = fmaxf(log_forget + m_old, log_in);
    keep = expf(log_forget + m_old - m_new);
    write = expf(log_in - m_new);
  };
  if (PIECES > 0) {
    constexpr int N = PIECES > 0 ? PIECES : 1, ROWS = N >= 4 ? 2 : 8 / N;      // state rows in flight per warp
    float4 q4[N], k4[N];
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int d = (n * 32 + lane) << 2;
      q4[n] = k4[n] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (d < D) {
        q4[n] = __ldcg(reinterpret_cast<const float4*>(q + d));
        k4[n] = __ldcg(reinterpret_cast<const float4*>(k + d));
      }
    }
    bool first = true;
    for (int v0 = warp; v0 <= V; v0 += DECODE_WARPS * ROWS) {
      float4 s[ROWS][N];
      float value[ROWS], sum[ROWS];
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        const int c = v0 + r * DECODE_WARPS;
        value[r] = c < V ? __ldcg(v + c) : 1.f;
#pragma unroll
        for (int n = 0; n < N; ++n) {
          const int d = (n * 32 + lane) << 2;
          s[r][n] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (c <= V && d < D) s[r][n] = __ldcg(reinterpret_cast<const float4*>(state + (size_t)c * D + d));
        }
      }
      if (first) gates();      // while the state is on its way
      first = false;
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        const int c = v0 + r * DECODE_WARPS;
        const float u = write * value[r];
        sum[r] = 0.f;
#pragma unroll
        for (int n = 0; n < N; ++n) {
          const int d = (n * 32 + lane) << 2;
          float4& x = s[r][n];
          x.x = fmaf(k4[n].x, u, keep * x.x); x.y = fmaf(k4[n].y, u, keep * x.y);
          x.z = fmaf(k4[n].z, u, keep * x.z); x.w = fmaf(k4[n].w, u, keep * x.w);
          sum[r] = fmaf(q4[n].x, x.x, sum[r]); sum[r] = fmaf(q4[n].y, x.y, sum[r]);
          sum[r] = fmaf(q4[n].z, x.z, sum[r]); sum[r] = fmaf(q4[n].w, x.w, sum[r]);
          if (c <= V && d < D) *reinterpret_cast<float4*>(state + (size_t)c * D + d) = x;
        }
      }
#pragma unroll
      for (int r = 0; r < ROWS; ++r) sum[r] = warp_sum(sum[r]);
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        const int c = v0 + r * DECODE_WARPS;
        if (lane == 0 && c <= V) shared[c] = sum[r] * p.q_scale;
      }
    }
    if (first) gates();        // a warp without a row of its own
  } else {
    gates();
    for (int c = warp; c <= V; c += DECODE_WARPS) {
      const float u = write * (c < V ? __ldcg(v + c) : 1.f);
      float sum = 0.f;
      for (int d = lane; d < D; d += 32) {
        float* s = state + (size_t)c * D + d;
        const float x = fmaf(__ldcg(k + d), u, keep * __ldcg(s));
        *s = x;
        sum = fmaf(__ldcg(q + d), x, sum);
      }
      sum = warp_sum(sum);
      if (lane == 0) shared[c] = sum * p.q_scale;
    }
  }
  __syncthreads();
  if (threadIdx.x == 0) p.maxima[slot_head] = m_new;      // every thread read the old one before the barrier
  const float inverse = 1.f / (fmaxf(fabsf(shared[V]), expf(-m_new)) + p.guard);
  float sq = 0.f;
  for (int c = threadIdx.x; c < V; c += DECODE_THREADS) {
    const float o = shared[c] * inverse;
    sq = fmaf(o, o, sq);
  }
  const float factor = inverse / sqrtf(block_sum(sq, scratch) / (float)V + p.eps);
  for (int c = threadIdx.x; c < V; c += DECODE_THREADS) {
    const float g = __ldcg(p.gate + row * p.gate_stride + (size_t)head * V + c);
    out[row * p.heads * V + (size_t)head * V + c] = from_float<T>(shared[c] * factor * p.weight[head * V + c] * sigmoid(g));
  }
}

// ------------------------------------------------------------------ gates of longer segments
constexpr int GATE_THREADS = 1024;
constexpr int GATE_WARPS = GATE_THREADS / 32;

// grid: (segments, heads).  1,024 tokens per turn.
__global__ void __launch_bounds__(GATE_THREADS)
matrix_memory_gates_kernel(MemoryArgs p) {
  __shared__ float total_a[GATE_WARPS], total_b[GATE_WARPS], last[GATE_WARPS];
  const int seg = blockIdx.x, head = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const size_t slot_head = (size_t)p.seg_slot[seg] * p.heads + head;
  const size_t row0 = p.seg_q_start[seg];
  const int q_len = p.seg_q_len[seg];
  const float i_bias = p.i_bias[head], f_bias = p.f_bias[head];
  // The recurrence behind this kernel is few blocks that run long: brought in while the product in front of this
  // kernel still fills the SMs, they would land several to an SM.  So the trigger comes after the wait.
  pdl_wait();
  pdl_trigger();
  float before = __ldcg(p.maxima + slot_head);       // m ahead of this turn's tokens
  float i_next = 0.f, f_next = 0.f;
  auto ask = [&](int t) {
    if (t < q_len) {
      i_next = __ldcg(p.i_raw + (row0 + t) * p.i_stride + head);
      f_next = __ldcg(p.f_raw + (row0 + t) * p.f_stride + head);
    }
  };
  ask(threadIdx.x);
  for (int t0 = 0; t0 < q_len; t0 += GATE_THREADS) {
    const int t = t0 + threadIdx.x;
    float log_in = -INFINITY, log_forget = 0.f;      // a place without a token changes nothing
    if (t < q_len) {
      log_in = capped(i_next + i_bias, p.cap);
      log_forget = log_sigmoid(capped(f_next + f_bias, p.cap));
    }
    ask(t + GATE_THREADS);
    // inclusive scan of the maps m -> max(a + m, b), earlier tokens first
    float a = log_forget, b = log_in;
#pragma unroll
    for (int step = 1; step < 32; step <<= 1) {
      const float a_up = __shfl_up_sync(0xffffffffu, a, step), b_up = __shfl_up_sync(0xffffffffu, b, step);
      if (lane >= step) {
        b = fmaxf(b_up + a, b);
        a += a_up;
      }
    }
    if (lane == 31) {
      total_a[warp] = a;
      total_b[warp] = b;
    }
    __syncthreads();
    float carried = before;
    for (int w = 0; w < warp; ++w) carried = fmaxf(total_a[w] + carried, total_b[w]);
    const float m = fmaxf(a + carried, b);
    if (lane == 31) last[warp] = m;
    __syncthreads();
    float m_before = __shfl_up_sync(0xffffffffu, m, 1);
    if (lane == 0) m_before = warp > 0 ? last[warp - 1] : before;
    if (t < q_len)
      p.coef[(row0 + t) * p.heads + head] = make_float4(expf(log_forget + m_before - m), expf(log_in - m), expf(-m), 0.f);
    before = last[GATE_WARPS - 1];
    __syncthreads();
  }
  if (threadIdx.x == 0) p.maxima[slot_head] = before;
}

// ------------------------------------------------------------------ the recurrence of longer segments
// grid: (segments, heads, blocks of state rows).  A group of SL lanes holds C rows of the head's transposed state
// (value channels, the last one the normaliser's), each lane E key channels of them in interleaved pieces of four.
// Reads are summed over the lanes for TB tokens at once; the updates need no sum.  WIDE: rows are staged in 16-byte
// pieces (sizes and strides multiples of four floats, pointers aligned).
template <int E, int SL, int C, bool WIDE, int THREADS>
__global__ void __launch_bounds__(THREADS)
matrix_memory_scan_kernel(MemoryArgs p) {
  pdl_trigger();
  extern __shared__ __align__(16) float shared[];
  constexpr int TB = 4, GROUPS = THREADS / SL, COLS = GROUPS * C, N = TB * C;
  constexpr int TOKENS = SL == 32 ? 16 : 32;      // tokens staged at once
  constexpr int pitch = E * SL;                   // staged rows of keys and queries, filled up with zeros
  constexpr int COEF = 4;
  constexpr int buffer = TOKENS * (2 * pitch + COLS + COEF);
  const int D = p.dim, V = p.vdim;
  const int seg = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * COLS;
  const int lane = threadIdx.x & 31, s = threadIdx.x % SL, group = threadIdx.x / SL;
  const int q_start = p.seg_q_start[seg], q_len = p.seg_q_len[seg];
  float* state = p.states + ((size_t)p.seg_slot[seg] * p.heads + head) * (size_t)(V + 1) * D;

  // what no copy overwrites: zeros behind the rows' D entries, the normaliser's value of one, zeros behind it
  if (D < pitch) {
    for (int idx = threadIdx.x; idx < 4 * TOKENS * (pitch - D); idx += THREADS) {
      const int r = idx / (pitch - D), d = D + idx - r * (pitch - D);
      shared[(r / (2 * TOKENS)) * buffer + (r % (2 * TOKENS)) * pitch + d] = 0.f;
    }
  }
  if (col0 + COLS > V) {
    for (int idx = threadIdx.x; idx < 2 * TOKENS * COLS; idx += THREADS) {
      const int which = idx / (TOKENS * COLS), at = idx - which * TOKENS * COLS, c = at % COLS;
      if (col0 + c >= V) shared[which * buffer + 2 * TOKENS * pitch + at] = col0 + c == V ? 1.f : 0.f;
    }
  }
  pdl_wait();
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
        copy_async_16(k_rows + t * pitch + d, p.k + (row0 + t) * p.k_stride + (size_t)head * D + d);
        copy_async_16(q_rows + t * pitch + d, p.q + (row0 + t) * p.q_stride + (size_t)head * D + d);
      }
      constexpr int V_PIECES = (COLS + 3) / 4;
      for (int idx = threadIdx.x; idx < tokens * V_PIECES; idx += THREADS) {
        const int t = idx / V_PIECES, c = (idx - t * V_PIECES) << 2;
        if (col0 + c < V) copy_async_16(v_rows + t * COLS + c, p.v + (row0 + t) * p.v_stride + (size_t)head * V + col0 + c);
      }
    } else {
      for (int idx = threadIdx.x; idx < tokens * D; idx += THREADS) {
        const int t = idx / D, d = idx - t * D;
        copy_async_4(k_rows + t * pitch + d, p.k + (row0 + t) * p.k_stride + (size_t)head * D + d);
        copy_async_4(q_rows + t * pitch + d, p.q + (row0 + t) * p.q_stride + (size_t)head * D + d);
      }
      for (int idx = threadIdx.x; idx < tokens * COLS; idx += THREADS) {
        const int t = idx / COLS, c = idx - t * COLS;
        if (col0 + c < V) copy_async_4(v_rows + idx, p.v + (row0 + t) * p.v_stride + (size_t)head * V + col0 + c);
      }
    }
    if (threadIdx.x < tokens)
      copy_async_16(coef + threadIdx.x * COEF, reinterpret_cast<const float*>(p.coef + (row0 + threadIdx.x) * p.heads + head));
    copy_async_commit();
    if (tokens % TB != 0) {      // the rest of the last block of tokens: kept as it is, nothing written
      const int fill = TB - tokens % TB;
      for (int idx = threadIdx.x; idx < fill * pitch; idx += THREADS) k_rows[tokens * pitch + idx] = q_rows[tokens * pitch + idx] = 0.f;
      for (int idx = threadIdx.x; idx < fill * COLS; idx += THREADS) v_rows[tokens * COLS + idx] = 0.f;
      for (int idx = threadIdx.x; idx < fill * COEF; idx += THREADS) coef[tokens * COEF + idx] = idx % COEF == 0 ? 1.f : 0.f;
    }
  };
  stage(0, 0);
  auto entry = [&](int i) { return (((i >> 2) * SL + s) << 2) + (i & 3); };      // key channel of a lane's i-th number
  float S[C][E];
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int column = col0 + group * C + c;
    const bool mine = column <= V;
    const float* src = state + (size_t)(mine ? column : 0) * D;
    if (WIDE) {
#pragma unroll
      for (int i = 0; i < E; i += 4) {
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (mine && entry(i) < D) x = __ldcg(reinterpret_cast<const float4*>(src + entry(i)));
        S[c][i] = x.x; S[c][i + 1] = x.y; S[c][i + 2] = x.z; S[c][i + 3] = x.w;
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
    const float* coef = v_rows + TOKENS * COLS;
    for (int t = 0; t < tokens; t += TB) {
      float read[N];
#pragma unroll
      for (int n = 0; n < TB; ++n) {
        const float2 gate = *reinterpret_cast<const float2*>(coef + (t + n) * COEF);      // keep, write
        float u[C];
#pragma unroll
        for (int c = 0; c < C; ++c) {
          u[c] = gate.y * v_rows[(t + n) * COLS + group * C + c];
          read[n * C + c] = 0.f;
        }
#pragma unroll
        for (int i = 0; i < E; i += 4) {
          const float4 k4 = *reinterpret_cast<const float4*>(k_rows + (t + n) * pitch + entry(i));
          const float4 q4 = *reinterpret_cast<const float4*>(q_rows + (t + n) * pitch + entry(i));
#pragma unroll
          for (int c = 0; c < C; ++c) {
            float sum = read[n * C + c];
            S[c][i] = fmaf(k4.x, u[c], gate.x * S[c][i]);
            sum = fmaf(q4.x, S[c][i], sum);
            S[c][i + 1] = fmaf(k4.y, u[c], gate.x * S[c][i + 1]);
            sum = fmaf(q4.y, S[c][i + 1], sum);
            S[c][i + 2] = fmaf(k4.z, u[c], gate.x * S[c][i + 2]);
            sum = fmaf(q4.z, S[c][i + 2], sum);
            S[c][i + 3] = fmaf(k4.w, u[c], gate.x * S[c][i + 3]);
            read[n * C + c] = fmaf(q4.w, S[c][i + 3], sum);
          }
        }
      }
      const int first = spread_sums<N, SL>(read, lane);
      constexpr int HELD = N > SL ? N / SL : 1;
      if (N >= SL || (s & (SL / N - 1)) == 0) {
#pragma unroll
        for (int i = 0; i < HELD; ++i) {
          const int number = first + i, n = number / C, column = col0 + group * C + number % C;
          if (t + n < tokens && column <= V) {
            const size_t row_head = (size_t)(q_start + t0 + t + n) * p.heads + head;
            if (column < V) p.reads[row_head * V + column] = read[i] * p.q_scale;
            else p.norms[row_head] = read[i] * p.q_scale;
          }
        }
      }
    }
    __syncthreads();      // the next turn of the loop stages into this buffer
  }
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int column = col0 + group * C + c;
    if (column > V) continue;
    float* dst = state + (size_t)column * D;
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

template <int E, int SL, int C, bool WIDE, int THREADS = 128>
static int launch_scan(const MemoryArgs& p, int segments, cudaStream_t stream) {
  constexpr int COLS = THREADS / SL * C, TOKENS = SL == 32 ? 16 : 32;
  constexpr size_t shared = sizeof(float) * 2 * (size_t)TOKENS * (2 * E * SL + COLS + 4);
  static_assert(shared <= 227 * 1024, "staging buffers");
  auto kernel = matrix_memory_scan_kernel<E, SL, C, WIDE, THREADS>;
  if (shared > 48 * 1024) {
    cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared);
    if (err != cudaSuccess) return (int)err;
  }
  launch_kernel(kernel, dim3(segments, p.heads, (p.vdim + 1 + COLS - 1) / COLS), dim3(THREADS), shared, stream, p);
  return launch_status();
}

// ------------------------------------------------------------------ chunks on the tensor cores
constexpr int CHUNK = 64;         // tokens
constexpr int CHUNK_COLS = 16;    // value channels of a block of the sequential kernel
constexpr int CHUNK_PITCH = CHUNK_COLS + 8;

__device__ __forceinline__ uint2 pack4(float4 x) { return make_uint2(pack_bf16(x.x, x.y), pack_bf16(x.z, x.w)); }

// grid: (chunks, heads, segments)
template <int D>
__global__ void __launch_bounds__(128)
matrix_memory_pairs_kernel(MemoryArgs p) {
  constexpr int PITCH = D + 8;
  extern __shared__ __align__(16) uint8_t raw[];
  bf16* q_tile = reinterpret_cast<bf16*>(raw);               // [64][PITCH]
  bf16* k_tile = q_tile + CHUNK * PITCH;
  float (*decay)[CHUNK + 1] = reinterpret_cast<float (*)[CHUNK + 1]>(k_tile + CHUNK * PITCH);
  __shared__ float keep[CHUNK], write[CHUNK];
  const int head = blockIdx.y, seg = blockIdx.z, V = p.vdim;
  const int t0 = blockIdx.x * CHUNK, count = min(CHUNK, p.seg_q_len[seg] - t0);
  if (count <= 0) return;
  const size_t row0 = (size_t)p.seg_q_start[seg] + t0;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  pdl_wait();
  if (threadIdx.x < CHUNK) {      // a place without a token keeps everything and writes nothing
    float2 gate = make_float2(1.f, 0.f);
    if (threadIdx.x < count) gate = __ldcg(reinterpret_cast<const float2*>(p.coef + (row0 + threadIdx.x) * p.heads + head));
    keep[threadIdx.x] = gate.x;
    write[threadIdx.x] = gate.y;
  }
  for (int idx = threadIdx.x; idx < CHUNK * (D / 4); idx += 128) {
    const int r = idx / (D / 4), d = (idx - r * (D / 4)) << 2;
    uint2 q2 = make_uint2(0u, 0u), k2 = q2;
    if (r < count) {
      const size_t at = (row0 + r) * p.heads * D + (size_t)head * D + d;
      q2 = pack4(__ldcg(reinterpret_cast<const float4*>(p.q + (row0 + r) * p.q_stride + (size_t)head * D + d)));
      k2 = pack4(__ldcg(reinterpret_cast<const float4*>(p.k + (row0 + r) * p.k_stride + (size_t)head * D + d)));
      *reinterpret_cast<uint2*>(p.q16 + at) = q2;
      *reinterpret_cast<uint2*>(p.k16 + at) = k2;
    }
    *reinterpret_cast<uint2*>(q_tile + r * PITCH + d) = q2;
    *reinterpret_cast<uint2*>(k_tile + r * PITCH + d) = k2;
  }
  for (int idx = threadIdx.x; idx < count * (V / 4); idx += 128) {
    const int r = idx / (V / 4), c = (idx - r * (V / 4)) << 2;
    *reinterpret_cast<uint2*>(p.v16 + (row0 + r) * p.heads * V + (size_t)head * V + c) =
        pack4(__ldcg(reinterpret_cast<const float4*>(p.v + (row0 + r) * p.v_stride + (size_t)head * V + c)));
  }
  __syncthreads();
  // a thread per column of D: its writing token's share at every later token
  if (threadIdx.x < CHUNK) {
    const int s = threadIdx.x;
    float x = write[s];
    for (int t = 0; t < CHUNK; ++t) {
      if (t > s) x *= keep[t];
      decay[t][s] = t >= s ? x : 0.f;
    }
    if (s < count) p.factors[(row0 + s) * p.heads + head].x = x;      // places behind the last token keep it
  } else if (threadIdx.x == CHUNK) {
    float x = 1.f;
    for (int t = 0; t < count; ++t) {
      x *= keep[t];
      p.factors[(row0 + t) * p.heads + head].y = x;
    }
  }
  uint32_t q_frag[D / 16][4];
#pragma unroll
  for (int ks = 0; ks < D / 16; ++ks)
    ldmatrix_x4(q_frag[ks], q_tile + (warp * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * PITCH + (ks * 2 + (lane >> 4)) * 8);
  float s[CHUNK / 8][4];
  padded_qk<D, CHUNK / 8>(s, q_frag, k_tile, lane);
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int t = warp * 16 + (lane >> 2) + 8 * i;
    if (t >= count) continue;
    float* dst = p.pairs + ((row0 + t) * p.heads + head) * CHUNK;
#pragma unroll
    for (int j = 0; j < CHUNK / 8; ++j) {
      const int c = j * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(dst + c) = make_float2(s[j][2 * i] * decay[t][c], s[j][2 * i + 1] * decay[t][c + 1]);
    }
  }
}

// the three bfloat16 parts of a pair of numbers
__device__ __forceinline__ void split_pair(float x, float y, uint32_t* part) {
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    const __nv_bfloat162 rounded = __floats2bfloat162_rn(x, y);
    part[i] = *reinterpret_cast<const uint32_t*>(&rounded);
    const float2 back = __bfloat1622float2(rounded);
    x -= back.x;
    y -= back.y;
  }
}

// c[0 .. 3] (four blocks of 8 columns) += a * tile, tile: 16 rows from `row` of a [..][CHUNK_PITCH] tile
__device__ __forceinline__ void mma_cols(float (*c)[4], const uint32_t* a, const bf16* tile, int row, int lane) {
#pragma unroll
  for (int dp = 0; dp < CHUNK_COLS / 16; ++dp) {
    uint32_t b[4];
    ldmatrix_x4_trans(b, tile + (row + (lane & 7) + (((lane >> 3) & 1) << 3)) * CHUNK_PITCH + (dp * 2 + (lane >> 4)) * 8);
    mma_bf16(c[2 * dp], a, b[0], b[1]);
    mma_bf16(c[2 * dp + 1], a, b[2], b[3]);
  }
}

// grid: (segments, heads, blocks of 32 state rows).  Warp w keeps the key channels w D / 4 .. of the state.
template <int D>
__global__ void __launch_bounds__(128)
matrix_memory_chunks_kernel(MemoryArgs p) {
  pdl_trigger();
  constexpr int PITCH = D + 8, MT = D / 64, NT = CHUNK_COLS / 8, PIECES = D / 8;
  extern __shared__ __align__(16) uint8_t raw[];
  bf16* qk_tiles = reinterpret_cast<bf16*>(raw);                       // 2 x (queries, keys) [64][PITCH]
  bf16* v_tiles = qk_tiles + 4 * CHUNK * PITCH;                         // 2 x [64][CHUNK_PITCH]
  bf16* s_parts = v_tiles + 2 * CHUNK * CHUNK_PITCH;                    // 3 x [D][CHUNK_PITCH]
  bf16* w_parts = s_parts + 3 * D * CHUNK_PITCH;                        // 3 x [64][CHUNK_PITCH]
  float2* factors = reinterpret_cast<float2*>(w_parts + 3 * CHUNK * CHUNK_PITCH);      // 2 x [64]
  const int seg = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * CHUNK_COLS, V = p.vdim;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int q_start = p.seg_q_start[seg], q_len = p.seg_q_len[seg];
  float* state = p.states + ((size_t)p.seg_slot[seg] * p.heads + head) * (size_t)(V + 1) * D;
  // value channels beyond the last: the normaliser's is one, the others zero; no copy overwrites them
  for (int idx = threadIdx.x; idx < 2 * CHUNK * CHUNK_COLS; idx += 128) {
    const int r = idx / CHUNK_COLS, c = idx - r * CHUNK_COLS;
    if (col0 + c >= V) v_tiles[r * CHUNK_PITCH + c] = __float2bfloat16_rn(col0 + c == V ? 1.f : 0.f);
  }
  pdl_wait();
  auto stage = [&](int t0, int which) {
    const int count = min(CHUNK, q_len - t0);
    const size_t row0 = (size_t)q_start + t0;
    bf16* q_tile = qk_tiles + which * 2 * CHUNK * PITCH;
    bf16* k_tile = q_tile + CHUNK * PITCH;
    for (int idx = threadIdx.x; idx < CHUNK * PIECES; idx += 128) {
      const int r = idx / PIECES, c = (idx - r * PIECES) * 8;
      const bool valid = r < count;
      const size_t at = valid ? (row0 + r) * p.heads * D + (size_t)head * D + c : 0;
      cp_async_16(q_tile + r * PITCH + c, p.q16 + at, valid);
      cp_async_16(k_tile + r * PITCH + c, p.k16 + at, valid);
    }
    for (int idx = threadIdx.x; idx < CHUNK * (CHUNK_COLS / 8); idx += 128) {
      const int r = idx / (CHUNK_COLS / 8), c = (idx - r * (CHUNK_COLS / 8)) * 8;
      if (col0 + c >= V) continue;
      const bool valid = r < count;
      cp_async_16(v_tiles + (which * CHUNK + r) * CHUNK_PITCH + c,
                  p.v16 + (valid ? (row0 + r) * p.heads * V + (size_t)head * V + col0 + c : 0), valid);
    }
    if (threadIdx.x < CHUNK) {      // a place without a token writes nothing
      const bool valid = threadIdx.x < count;
      copy_async_8(factors + which * CHUNK + threadIdx.x, p.factors + (valid ? (row0 + threadIdx.x) * p.heads + head : 0), valid);
    }
    cp_async_commit();
  };
  stage(0, 0);
  float S[MT][NT][4];      // accumulators: key channel (row) lane / 4 + 8 (e / 2), value channel (column) 2 (lane % 4) + e % 2
  auto place = [&](int mt, int nt, int e, int* d, int* c) {
    *d = warp * (D / 4) + mt * 16 + (lane >> 2) + 8 * (e >> 1);
    *c = col0 + nt * 8 + (lane & 3) * 2 + (e & 1);
  };
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        int d, c;
        place(mt, nt, e, &d, &c);
        S[mt][nt][e] = c <= V ? __ldcg(state + (size_t)c * D + d) : 0.f;
      }
  int which = 0;
  for (int t0 = 0; t0 < q_len; t0 += CHUNK, which ^= 1) {
    const int count = min(CHUNK, q_len - t0);
    const size_t row0 = (size_t)q_start + t0;
    cp_async_wait<0>();
    __syncthreads();      // this chunk is here, and everybody is done with the one before
    if (t0 + CHUNK < q_len) stage(t0 + CHUNK, which ^ 1);
    const bf16* q_tile = qk_tiles + which * 2 * CHUNK * PITCH;
    const bf16* k_tile = q_tile + CHUNK * PITCH;
    const bf16* v_tile = v_tiles + which * CHUNK * CHUNK_PITCH;
    const float2* factor = factors + which * CHUNK;
    // this warp's rows of A, asked for early: keys up to the rows' own chunk part only
    const int r0 = warp * 16 + (lane >> 2);
    const float* a_row[2] = {p.pairs + ((row0 + r0) * p.heads + head) * CHUNK + (lane & 3) * 2,
                             p.pairs + ((row0 + r0 + 8) * p.heads + head) * CHUNK + (lane & 3) * 2};
    float2 a_pair[CHUNK / 16][4];
#pragma unroll
    for (int ks = 0; ks < CHUNK / 16; ++ks)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        a_pair[ks][e] = make_float2(0.f, 0.f);
        if (ks <= warp && r0 + 8 * (e & 1) < count)
          a_pair[ks][e] = __ldcg(reinterpret_cast<const float2*>(a_row[e & 1] + ks * 16 + 8 * (e >> 1)));
      }
    // the state and the weighed values in parts
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          uint32_t part[3];
          split_pair(S[mt][nt][2 * i], S[mt][nt][2 * i + 1], part);
          int d, c;
          place(mt, nt, 2 * i, &d, &c);
#pragma unroll
          for (int n = 0; n < 3; ++n)
            *reinterpret_cast<uint32_t*>(s_parts + (n * D + d) * CHUNK_PITCH + (c - col0)) = part[n];
        }
    for (int idx = threadIdx.x; idx < CHUNK * (CHUNK_COLS / 2); idx += 128) {
      const int r = idx / (CHUNK_COLS / 2), c = (idx - r * (CHUNK_COLS / 2)) * 2;
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(v_tile + r * CHUNK_PITCH + c));
      const float weight = factor[r].x;
      uint32_t part[3];
      split_pair(weight * v.x, weight * v.y, part);
#pragma unroll
      for (int n = 0; n < 3; ++n) *reinterpret_cast<uint32_t*>(w_parts + (n * CHUNK + r) * CHUNK_PITCH + c) = part[n];
    }
    __syncthreads();
    // reads: of the state before the chunk, then of the chunk's own tokens; a sum per part (short chains of products)
    float o[3][NT][4];
#pragma unroll
    for (int n = 0; n < 3; ++n)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) o[n][nt][0] = o[n][nt][1] = o[n][nt][2] = o[n][nt][3] = 0.f;
    if (warp * 16 < count) {
#pragma unroll
      for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t a[4];
        ldmatrix_x4(a, q_tile + (warp * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * PITCH + (ks * 2 + (lane >> 4)) * 8);
#pragma unroll
        for (int n = 0; n < 3; ++n) mma_cols(o[n], a, s_parts + n * D * CHUNK_PITCH, ks * 16, lane);
      }
      const float before[2] = {factor[r0].y, factor[r0 + 8].y};
#pragma unroll
      for (int n = 0; n < 3; ++n)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) o[n][nt][e] *= before[e >> 1];
#pragma unroll
      for (int ks = 0; ks < CHUNK / 16; ++ks) {
        if (ks > warp) continue;
        uint32_t part[4][3];
#pragma unroll
        for (int e = 0; e < 4; ++e) split_pair(a_pair[ks][e].x, a_pair[ks][e].y, part[e]);
#pragma unroll
        for (int n = 0; n < 3; ++n) {
          const uint32_t a[4] = {part[0][n], part[1][n], part[2][n], part[3][n]};
          mma_cols(o[n], a, v_tile, ks * 16, lane);
        }
      }
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[0][nt][e] += o[1][nt][e] + o[2][nt][e];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        if (r0 + 8 * i >= count) continue;
        const size_t row_head = (row0 + r0 + 8 * i) * p.heads + head;
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const int c = col0 + nt * 8 + (lane & 3) * 2;
          if (c < V)
            *reinterpret_cast<float2*>(p.reads + row_head * V + c) = make_float2(o[0][nt][2 * i] * p.q_scale, o[0][nt][2 * i + 1] * p.q_scale);
          else if (c == V)
            p.norms[row_head] = o[0][nt][2 * i] * p.q_scale;
        }
      }
    }
    // the state behind the chunk
    const float kept = factor[count - 1].y;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[mt][nt][e] *= kept;
#pragma unroll
      for (int ks = 0; ks < CHUNK / 16; ++ks) {
        uint32_t a[4];      // keys transposed: channels are the product's rows
        ldmatrix_x4_trans(a, k_tile + (ks * 16 + ((lane >> 4) << 3) + (lane & 7)) * PITCH + warp * (D / 4) + mt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int n = 2; n >= 0; --n) mma_cols(S[mt], a, w_parts + n * CHUNK * CHUNK_PITCH, ks * 16, lane);
      }
    }
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        int d, c;
        place(mt, nt, e, &d, &c);
        if (c <= V) state[(size_t)c * D + d] = S[mt][nt][e];
      }
}

template <int D>
static int launch_chunks(const MemoryArgs& p, int segments, int max_q_len, cudaStream_t stream) {
  constexpr size_t shared = sizeof(bf16) * (size_t)(4 * CHUNK * (D + 8) + (2 * CHUNK + 3 * D + 3 * CHUNK) * CHUNK_PITCH) +
                            sizeof(float2) * 2 * CHUNK;
  static_assert(shared <= 227 * 1024, "tiles");
  constexpr size_t pairs_shared = sizeof(bf16) * (size_t)(2 * CHUNK * (D + 8)) + sizeof(float) * CHUNK * (CHUNK + 1);
  cudaError_t err = cudaFuncSetAttribute(matrix_memory_chunks_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared);
  if (err == cudaSuccess)
    err = cudaFuncSetAttribute(matrix_memory_pairs_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)pairs_shared);
  if (err != cudaSuccess) return (int)err;
  launch_kernel(matrix_memory_pairs_kernel<D>, dim3((max_q_len + CHUNK - 1) / CHUNK, p.heads, segments), dim3(128), pairs_shared,
                stream, p);
  const int status = launch_status();
  if (status != MLR_OK) return status;
  launch_kernel(matrix_memory_chunks_kernel<D>, dim3(segments, p.heads, (p.vdim + CHUNK_COLS) / CHUNK_COLS), dim3(128), shared, stream, p);
  return launch_status();
}

// ------------------------------------------------------------------ normaliser, head norm, weight, gate
__device__ __forceinline__ void store4(float* dst, float4 y) { *reinterpret_cast<float4*>(dst) = y; }
__device__ __forceinline__ void store4(bf16* dst, float4 y) { *reinterpret_cast<uint2*>(dst) = pack4(y); }

// A warp per (row, head).  WIDE: at most 256 channels, in pieces of four (sizes, strides and pointers allow it).
template <typename T, bool WIDE>
__global__ void __launch_bounds__(128)
matrix_memory_finish_kernel(MemoryArgs p, T* __restrict__ out, long long items) {
  pdl_trigger();
  pdl_wait();
  const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (item >= items) return;
  const int lane = threadIdx.x & 31, V = p.vdim;
  const long long row = item / p.heads;
  const int head = (int)(item - row * p.heads);
  const float* reads = p.reads + item * V;
  const float* gate = p.gate + row * p.gate_stride + (size_t)head * V;
  const float* weight = p.weight + (size_t)head * V;
  const float inverse = 1.f / (fmaxf(fabsf(__ldcg(p.norms + item)), __ldcg(&p.coef[item].z)) + p.guard);
  if (WIDE) {
    float4 o[2], g[2];
    float sq = 0.f;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int c = (lane + 32 * j) * 4;
      o[j] = g[j] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < V) {
        o[j] = __ldcg(reinterpret_cast<const float4*>(reads + c));
        g[j] = __ldcg(reinterpret_cast<const float4*>(gate + c));
      }
      o[j].x *= inverse; o[j].y *= inverse; o[j].z *= inverse; o[j].w *= inverse;
      sq += fmaf(o[j].x, o[j].x, o[j].y * o[j].y) + fmaf(o[j].z, o[j].z, o[j].w * o[j].w);
    }
    const float factor = 1.f / sqrtf(warp_sum(sq) / (float)V + p.eps);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int c = (lane + 32 * j) * 4;
      if (c >= V) continue;
      const float4 w = *reinterpret_cast<const float4*>(weight + c);
      store4(out + item * V + c, make_float4(o[j].x * factor * w.x * sigmoid(g[j].x), o[j].y * factor * w.y * sigmoid(g[j].y),
                                             o[j].z * factor * w.z * sigmoid(g[j].z), o[j].w * factor * w.w * sigmoid(g[j].w)));
    }
    return;
  }
  constexpr int HELD = 8;      // channels a lane keeps in registers
  float o[HELD], g[HELD], sq = 0.f;
#pragma unroll
  for (int j = 0; j < HELD; ++j) {
    const int c = lane + 32 * j;
    o[j] = c < V ? __ldcg(reads + c) * inverse : 0.f;
    g[j] = c < V ? __ldcg(gate + c) : 0.f;
    sq = fmaf(o[j], o[j], sq);
  }
  for (int c = lane + 32 * HELD; c < V; c += 32) {
    const float x = __ldcg(reads + c) * inverse;
    sq = fmaf(x, x, sq);
  }
  const float factor = 1.f / sqrtf(warp_sum(sq) / (float)V + p.eps);
  T* dst = out + item * V;
#pragma unroll
  for (int j = 0; j < HELD; ++j) {
    const int c = lane + 32 * j;
    if (c < V) dst[c] = from_float<T>(o[j] * factor * weight[c] * sigmoid(g[j]));
  }
  for (int c = lane + 32 * HELD; c < V; c += 32)
    dst[c] = from_float<T>(__ldcg(reads + c) * inverse * factor * weight[c] * sigmoid(__ldcg(gate + c)));
}

static bool chunks_fit(int dim, int vdim) { return (dim == 64 || dim == 128) && vdim % 8 == 0; }

template <typename T>
static int launch_memory(const MemoryArgs& p, T* out, int rows, int segments, int max_q_len, bool wide, cudaStream_t stream) {
  const int D = p.dim;
  if (max_q_len == 1) {
    const dim3 grid(segments, p.heads);
    const size_t shared = sizeof(float) * (size_t)(p.vdim + 1);
    if (!wide) launch_kernel(matrix_memory_decode_kernel<T, 0>, grid, dim3(DECODE_THREADS), shared, stream, p, out);
    else if (D <= 128) launch_kernel(matrix_memory_decode_kernel<T, 1>, grid, dim3(DECODE_THREADS), shared, stream, p, out);
    else if (D <= 256) launch_kernel(matrix_memory_decode_kernel<T, 2>, grid, dim3(DECODE_THREADS), shared, stream, p, out);
    else launch_kernel(matrix_memory_decode_kernel<T, 4>, grid, dim3(DECODE_THREADS), shared, stream, p, out);
    return launch_status();
  }
  if (p.coef == nullptr || p.reads == nullptr || p.norms == nullptr) return MLR_BAD_SIZE;
  launch_kernel(matrix_memory_gates_kernel, dim3(segments, p.heads), dim3(GATE_THREADS), 0, stream, p);
  int status = launch_status();
  if (status != MLR_OK) return status;
  if (p.pairs != nullptr) {
    if (!wide || !chunks_fit(D, p.vdim)) return MLR_BAD_SIZE;
    status = D == 64 ? launch_chunks<64>(p, segments, max_q_len, stream) : launch_chunks<128>(p, segments, max_q_len, stream);
  } else if (wide) {
    if (D <= 32) status = launch_scan<4, 8, 1, true>(p, segments, stream);
    else if (D <= 64) status = launch_scan<4, 16, 1, true>(p, segments, stream);
    else if (D <= 128) status = launch_scan<8, 16, 2, true>(p, segments, stream);
    else if (D <= 256) status = launch_scan<8, 32, 2, true>(p, segments, stream);
    else status = launch_scan<16, 32, 2, true>(p, segments, stream);
  } else {
    if (D <= 32) status = launch_scan<4, 8, 1, false>(p, segments, stream);
    else if (D <= 128) status = launch_scan<16, 8, 1, false>(p, segments, stream);
    else status = launch_scan<16, 32, 1, false>(p, segments, stream);
  }
  if (status != MLR_OK) return status;
  const long long items = (long long)rows * p.heads;
  auto aligned = [](const void* ptr) { return (reinterpret_cast<uintptr_t>(ptr) & 15) == 0; };
  const bool pieces = p.vdim % 4 == 0 && p.vdim <= 256 && p.gate_stride % 4 == 0 && aligned(p.gate) && aligned(p.reads) &&
                      aligned(p.weight) && aligned(out);
  launch_kernel(pieces ? matrix_memory_finish_kernel<T, true> : matrix_memory_finish_kernel<T, false>,
                dim3((unsigned)((items + 3) / 4)), dim3(128), 0, stream, p, out, items);
  return launch_status();
}

}  // namespace mlr

using namespace mlr;

MLR_DEFINE_PDL_SWITCH

// Whether prompts of these head sizes can go through the tensor cores in chunks (with `pairs`).
MLR_EXPORT int mlr_matrix_memory_chunks_fit(int dim, int vdim) { return chunks_fit(dim, vdim); }

// q, k: float32 rows of heads * dim entries; v, gate: rows of heads * vdim; i_raw, f_raw: rows of `heads` entries (each
// with its own row stride); i_bias, f_bias: float32 [heads]; weight: float32 [heads * vdim]; coef: float32 scratch
// [rows, heads, 4], reads: [rows, heads, vdim], norms: [rows, heads] (all three null for steps of single rows); pairs:
// float32 scratch [rows, heads, 64 + 2] and packed: bfloat16 scratch [rows, heads, 2 dim + vdim] (both or neither: chunks
// on the tensor cores, or the token-by-token scan; 16-byte aligned); states:
// float32 [slots, heads, vdim + 1, dim], maxima: float32 [slots, heads]; out: [rows, heads * vdim] in `dtype`.
// max_q_len: the longest segment of the step.
MLR_EXPORT int mlr_matrix_memory(const float* q, long long q_stride, const float* k, long long k_stride, const float* v,
                                 long long v_stride, const float* i_raw, long long i_stride, const float* f_raw,
                                 long long f_stride, const float* gate, long long gate_stride, const float* i_bias,
                                 const float* f_bias, const float* weight, float* coef, float* reads, float* norms,
                                 float* pairs, void* packed, float* states, float* maxima, void* out, const int* seg_q_start, const int* seg_q_len,
                                 const int* seg_slot, int rows, int segments, int max_q_len, int heads, int dim, int vdim,
                                 float cap, float guard, float eps, float q_scale, int dtype, cudaStream_t stream) {
  if (segments == 0 || rows == 0) return MLR_OK;
  if (segments < 0 || rows < 0 || max_q_len <= 0 || heads <= 0 || dim <= 0 || vdim <= 0 || !(cap > 0.f)) return MLR_BAD_SIZE;
  if (dim > 512 || vdim > 4096 || heads > 65535 || segments > 65535) return MLR_TOO_LARGE;
  bf16* q16 = (bf16*)packed;
  bf16* k16 = q16 == nullptr ? nullptr : q16 + (size_t)rows * heads * dim;
  bf16* v16 = q16 == nullptr ? nullptr : k16 + (size_t)rows * heads * dim;
  if ((pairs == nullptr) != (packed == nullptr)) return MLR_BAD_SIZE;
  MemoryArgs p{q, k, v, i_raw, f_raw, gate, q_stride, k_stride, v_stride, i_stride, f_stride, gate_stride, i_bias, f_bias,
               weight, reinterpret_cast<float4*>(coef), reads, norms, pairs,
               pairs == nullptr ? nullptr : reinterpret_cast<float2*>(pairs + (size_t)rows * heads * CHUNK), q16, k16, v16, states, maxima, seg_q_start, seg_q_len, seg_slot, heads,
               dim, vdim, cap, guard, eps, q_scale};
  auto multiple = [](long long n) { return n % 4 == 0; };
  auto aligned = [](const void* ptr) { return (reinterpret_cast<uintptr_t>(ptr) & 15) == 0; };
  if (!aligned(coef) || !aligned(pairs) || !aligned(packed)) return MLR_BAD_ALIGNMENT;
  const bool wide = multiple(dim) && multiple(vdim) && multiple(q_stride) && multiple(k_stride) && multiple(v_stride) &&
                    aligned(q) && aligned(k) && aligned(v) && aligned(states);
  if (dtype == MLR_F32) return launch_memory(p, (float*)out, rows, segments, max_q_len, wide, stream);
  if (dtype == MLR_BF16) return launch_memory(p, (bf16*)out, rows, segments, max_q_len, wide, stream);
  return MLR_BAD_DTYPE;
}
