// Grouped-query softmax attention with shaped scores, on the tensor cores (bfloat16, mma.sync m16n8k16), over keys
// that are also the values or over values of the keys' size of their own.  Per head h, query position i and key
// position j:
//
//   x = softcap * tanh(q . k * scale / softcap)  (or q . k * scale without a cap)  - slope_h * (i - j)
//   visible: j <= i, j in i's own chunk (chunk > 0), i - j < window (window > 0)
//   out = sum_j e^x_j v_j / (sum_j e^x_j + e^sink_h), times sigmoid(gate) element by element
//
// Scores, cap, bias, softmax and sums are float32; the probabilities are rounded to bfloat16 for the second
// product.  Where keys are the values a key tile is fetched once and serves both products (OWN false); else a tile
// of keys and one of values lie side by side in shared memory.
//
// shaped_prefill_kernel  work item (64 query rows of a segment, head): tiles of 64 keys aligned to absolute
//                        positions, double-buffered with asynchronous copies, the tiles' places in the cache
//                        looked up once per tile.
// shaped_decode_kernel   one-row segments: the query heads of a key/value head (16 at a time) are the rows of
//                        the products; the visible keys are cut over CTAs, within a CTA each warp walks key
//                        tiles of 32 of its own; the warps' parts are merged in shared memory, the CTAs'
//                        parts by the last CTA to finish, in the order of the keys.  In a step of decoded
//                        tokens only the kernel takes the new token's key from the projection and stores it
//                        into its page itself.
#include "mma_attention.cuh"

namespace mlr {

constexpr float LOG2E = 1.4426950408889634f;

// 2^x by the hardware's approximate instruction (about 2 ulp); minus infinity gives 0.
__device__ __forceinline__ float exp2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct ShapedArgs {
  const bf16* q; long long q_stride;             // rows of heads * D
  const bf16* fresh; long long fresh_stride;     // decode: rows of kv_heads * D with the new keys, or null (already cached)
  const long long* slots;                        // decode with fresh: where each row's key goes
  bf16* pool;                                    // [pages, kv_heads, page_size, D]
  const bf16* values;                            // the same for values of their own, or null
  bf16* out;                                     // [rows, heads * D]
  const bf16* gate; long long gate_stride;       // rows of heads * D, or null
  const float *slopes, *sinks;                   // [heads] or null
  const int *tile_seg, *tile_row0;               // prefill
  const int* decode_seg;                         // decode: segments, or null (segment i is i)
  const int *seg_q_start, *seg_q_len, *seg_pos0, *block_table, *seg_slot;
  int table_width, heads, kv_heads, page_size, page_shift, window, chunk;
  float in_scale, out_scale;                     // capped: scale / cap and cap * log2(e); else scale * log2(e) and 1
  int capped;
  float* partial; float2* limits; int* counters; int splits;     // decode
};

// tanh of every number of a fragment.  Small arguments (the usual case by far: a cap is chosen well above the
// scores) take the first terms of its Taylor series, whose error below 1/4 is under 3e-9; the choice is the
// warp's, so it costs one vote.
template <int N>
__device__ __forceinline__ void fragment_tanh(float (*s)[4]) {
  float top = 0.f;
#pragma unroll
  for (int j = 0; j < N; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) top = fmaxf(top, fabsf(s[j][e]));
  if (!__any_sync(0xffffffffu, top > 0.25f)) {
#pragma unroll
    for (int j = 0; j < N; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float t = s[j][e], t2 = t * t;
        float r = fmaf(t2, 62.f / 2835.f, -17.f / 315.f);
        r = fmaf(t2, r, 2.f / 15.f);
        r = fmaf(t2, r, -1.f / 3.f);
        s[j][e] = fmaf(t * t2, r, t);
      }
    return;
  }
#pragma unroll
  for (int j = 0; j < N; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      // 1 - 2 / (1 + e^(2|t|)), odd in t; the exponent is kept where the division is defined
      const float t = s[j][e];
      const float r = 1.f - __fdividef(2.f, 1.f + __expf(fminf(2.f * fabsf(t), 80.f)));
      s[j][e] = copysignf(r, t);
    }
}

// One warp's raw scores (rows r0 = lane / 4 and r0 + 8, NT blocks of 8 keys from key_base) to log2-domain
// shaped scores, then the online softmax step: probabilities in s, o rescaled.
template <int NT, int OT, bool MASKED>
__device__ __forceinline__ void shaped_softmax_step(float (*s)[4], float (*o)[4], float* m, float* l, int key_base,
                                                    const int* position, const int* limit_lo, const float* slope2,
                                                    const ShapedArgs& p, int lane) {
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) s[j][e] *= p.in_scale;
  if (p.capped) fragment_tanh<NT>(s);
  const int key_lane = key_base + (lane & 3) * 2;
  const float start[2] = {slope2[0] * (float)(key_lane - position[0]), slope2[1] * (float)(key_lane - position[1])};
  float tile_max[2] = {-INFINITY, -INFINITY};
#pragma unroll
  for (int j = 0; j < NT; ++j) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = e >> 1, step = j * 8 + (e & 1), key = key_lane + step;
      const float x = fmaf(s[j][e], p.out_scale, fmaf(slope2[i], (float)step, start[i]));
      s[j][e] = !MASKED || (key >= limit_lo[i] && key <= position[i]) ? x : -INFINITY;
      tile_max[i] = fmaxf(tile_max[i], s[j][e]);
    }
  }
  float alpha[2], row_sum[2] = {0.f, 0.f}, base[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    tile_max[i] = fmaxf(tile_max[i], __shfl_xor_sync(0xffffffffu, tile_max[i], 1));
    tile_max[i] = fmaxf(tile_max[i], __shfl_xor_sync(0xffffffffu, tile_max[i], 2));
    const float m_new = fmaxf(m[i], tile_max[i]);
    base[i] = m_new == -INFINITY ? 0.f : m_new;       // nothing visible yet: keep everything at zero
    alpha[i] = exp2_approx(m[i] - base[i]);                 // m = -inf gives 0
    m[i] = m_new;
  }
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      s[j][e] = exp2_approx(s[j][e] - base[e >> 1]);
      row_sum[e >> 1] += s[j][e];
    }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    row_sum[i] += __shfl_xor_sync(0xffffffffu, row_sum[i], 1);
    row_sum[i] += __shfl_xor_sync(0xffffffffu, row_sum[i], 2);
    l[i] = l[i] * alpha[i] + row_sum[i];
  }
#pragma unroll
  for (int t = 0; t < OT; ++t) {
    o[t][0] *= alpha[0]; o[t][1] *= alpha[0];
    o[t][2] *= alpha[1]; o[t][3] *= alpha[1];
  }
}

// Row of the pool (in units of D entries) that holds a key of one kv head, or -1.
__device__ __forceinline__ int pool_row(const ShapedArgs& p, const int* table, int key, int kv_head) {
  const int logical = p.page_shift >= 0 ? key >> p.page_shift : key / p.page_size;
  const int page = table[logical];
  if (page < 0) return -1;
  return (page * p.kv_heads + kv_head) * p.page_size + (key - logical * p.page_size);
}

__device__ __forceinline__ int lowest_visible(const ShapedArgs& p, int position) {
  int lo = p.chunk > 0 ? position / p.chunk * p.chunk : 0;
  if (p.window > 0) lo = max(lo, position - p.window + 1);
  return lo;
}

template <int D, bool OWN>
__global__ void __launch_bounds__(ATTN_THREADS, OWN ? 2 : D <= 64 ? 4 : 3)
shaped_prefill_kernel(const ShapedArgs p) {
  pdl_trigger();
  pdl_wait();
  constexpr int PITCH = D + 8, PIECES = D / 8, KINDS = OWN ? 2 : 1, TILE = TILE_KV * PITCH;
  extern __shared__ __align__(128) uint8_t attn_shared[];
  bf16* q_tile = reinterpret_cast<bf16*>(attn_shared);         // [64][PITCH]
  bf16* k_tiles = q_tile + TILE_Q * PITCH;                      // 2 x [64][PITCH] (keys, then values of their own)
  __shared__ int places[2][TILE_KV];                            // pool rows of a tile's keys, two tiles ahead

  const int head = blockIdx.y, kv_head = head / (p.heads / p.kv_heads);
  const int seg = p.tile_seg[blockIdx.x], row0 = p.tile_row0[blockIdx.x];      // the list is heaviest first
  const int q_start = p.seg_q_start[seg], q_len = p.seg_q_len[seg], pos0 = p.seg_pos0[seg];
  const int rows = min(TILE_Q, q_len - row0);
  const int* table = p.block_table + (size_t)p.seg_slot[seg] * p.table_width;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  const int first_pos = pos0 + row0, last_pos = first_pos + rows - 1;
  const int lowest = lowest_visible(p, first_pos);
  const int begin = lowest / TILE_KV, end = last_pos / TILE_KV;                // inclusive

  for (int item = threadIdx.x; item < TILE_Q * PIECES; item += ATTN_THREADS) {
    const int r = item / PIECES, c = item - r * PIECES;
    const bool valid = r < rows;
    cp_async_16(q_tile + r * PITCH + c * 8,
                valid ? p.q + (size_t)(q_start + row0 + r) * p.q_stride + head * D + c * 8 : p.q, valid);
  }
  auto look_up = [&](int t) {
    if (threadIdx.x < TILE_KV) {
      const int key = t * TILE_KV + threadIdx.x;
      places[t & 1][threadIdx.x] = key >= lowest && key <= last_pos ? pool_row(p, table, key, kv_head) : -1;
    }
  };
  auto fetch = [&](int t) {
    bf16* tile = k_tiles + (t & 1) * KINDS * TILE;
    for (int item = threadIdx.x; item < TILE_KV * PIECES; item += ATTN_THREADS) {
      const int r = item / PIECES, c = item - r * PIECES;
      const int row = places[t & 1][r];
      cp_async_16(tile + r * PITCH + c * 8, row >= 0 ? p.pool + (size_t)row * D + c * 8 : p.pool, row >= 0);
      if (OWN) cp_async_16(tile + TILE + r * PITCH + c * 8, row >= 0 ? p.values + (size_t)row * D + c * 8 : p.values, row >= 0);
    }
    cp_async_commit();
  };
  look_up(begin);
  look_up(begin + 1);
  __syncthreads();
  fetch(begin);

  int position[2], limit_lo[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = warp * 16 + (lane >> 2) + 8 * i;
    position[i] = r < rows ? first_pos + r : -1;                // rows past the segment see nothing
    limit_lo[i] = r < rows ? lowest_visible(p, first_pos + r) : 0;
  }
  // what all rows of the warp see (no mask needed) and what any of them sees
  const int warp_rows = min(16, rows - warp * 16);
  const int warp_first = first_pos + warp * 16, warp_last = warp_first + warp_rows - 1;
  const int any_lo = warp_rows > 0 ? lowest_visible(p, warp_first) : 0;
  const int all_lo = warp_rows > 0 ? lowest_visible(p, warp_last) : 0;
  const float slope = (p.slopes != nullptr ? p.slopes[head] : 0.f) * LOG2E;
  const float slope2[2] = {slope, slope};
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float o[D / 8][4];
#pragma unroll
  for (int t = 0; t < D / 8; ++t) o[t][0] = o[t][1] = o[t][2] = o[t][3] = 0.f;
  uint32_t q_frag[D / 16][4];

  for (int t = begin; t <= end; ++t) {
    if (t < end) {
      fetch(t + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    if (t + 2 <= end) look_up(t + 2);      // places of tile t were read before the barrier above
    if (t == begin) {
#pragma unroll
      for (int ks = 0; ks < D / 16; ++ks)
        ldmatrix_x4(q_frag[ks], q_tile + (warp * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * PITCH + (ks * 2 + (lane >> 4)) * 8);
    }
    const int key0 = t * TILE_KV, key_last = key0 + TILE_KV - 1;
    if (warp_rows > 0 && key0 <= warp_last && key_last >= any_lo) {
      const bf16* tile = k_tiles + (t & 1) * KINDS * TILE;
      float s[TILE_KV / 8][4];
      padded_qk<D, TILE_KV / 8>(s, q_frag, tile, lane);
      if (warp_rows == 16 && key_last <= warp_first && key0 >= all_lo)
        shaped_softmax_step<TILE_KV / 8, D / 8, false>(s, o, m, l, key0, position, limit_lo, slope2, p, lane);
      else
        shaped_softmax_step<TILE_KV / 8, D / 8, true>(s, o, m, l, key0, position, limit_lo, slope2, p, lane);
      padded_pv<D, TILE_KV / 8>(o, s, tile + (KINDS - 1) * TILE, lane);
    }
    __syncthreads();
  }

#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = warp * 16 + (lane >> 2) + 8 * i;
    if (r >= rows) continue;
    float factor = 1.f / l[i];
    if (p.sinks != nullptr) {
      const float sink = p.sinks[head] * LOG2E, top = fmaxf(m[i], sink), share = exp2_approx(m[i] - top);
      factor = share / fmaf(l[i], share, exp2_approx(sink - top));
    }
    const size_t row = (size_t)(q_start + row0 + r);
    const int column = head * D + (lane & 3) * 2;
    bf16* dst = p.out + row * p.heads * D + column;
    const bf16* gate = p.gate != nullptr ? p.gate + row * p.gate_stride + column : nullptr;
#pragma unroll
    for (int t = 0; t < D / 8; ++t) {
      float a = o[t][2 * i] * factor, b = o[t][2 * i + 1] * factor;
      if (gate != nullptr) {
        const uint32_t raw = __ldcg(reinterpret_cast<const unsigned int*>(gate + t * 8));
        const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw));
        a = __fdividef(a, 1.f + __expf(fminf(-g.x, 80.f)));
        b = __fdividef(b, 1.f + __expf(fminf(-g.y, 80.f)));
      }
      *reinterpret_cast<uint32_t*>(dst + t * 8) = pack_bf16(a, b);
    }
  }
}

constexpr int DEC_KEYS = 32;         // keys of a warp's tile
// tiles of a warp in shared memory: with values of their own and wide heads one, so that three blocks fit an SM
template <int D, bool OWN> constexpr int DEC_STAGES = OWN && D > 64 ? 1 : 2;
constexpr int DEC_ROWS = 16;         // query heads of one CTA
constexpr int DEC_MAX_SPLITS = 64;
constexpr int DEC_MIN_TILES = 4;     // key tiles a CTA takes at least (one per warp)

// grid: (items, kv heads * blocks of 16 query heads, splits)
template <int D, bool OWN>
__global__ void __launch_bounds__(ATTN_THREADS)
shaped_decode_kernel(const ShapedArgs p) {
  pdl_trigger();
  constexpr int PITCH = D + 8, PIECES = D / 8, KINDS = OWN ? 2 : 1, STAGES = DEC_STAGES<D, OWN>, TILE = DEC_KEYS * PITCH;
  constexpr int PER_LANE = DEC_KEYS * PIECES / 32;
  extern __shared__ __align__(128) uint8_t attn_shared[];
  bf16* q_tile = reinterpret_cast<bf16*>(attn_shared);                              // [16][PITCH]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  bf16* ring = q_tile + DEC_ROWS * PITCH + warp * STAGES * KINDS * TILE;            // this warp's tiles
  float* merged = reinterpret_cast<float*>(q_tile + DEC_ROWS * PITCH);              // [4][16][D] once the tiles are done
  __shared__ float warp_max_[ATTN_WARPS][DEC_ROWS], warp_sum_[ATTN_WARPS][DEC_ROWS];
  __shared__ int is_last;

  const int per = p.heads / p.kv_heads, blocks = (per + DEC_ROWS - 1) / DEC_ROWS;
  const int kv_head = blockIdx.y / blocks, block = blockIdx.y - kv_head * blocks;
  const int head0 = kv_head * per + block * DEC_ROWS;
  const int live = min(DEC_ROWS, per - block * DEC_ROWS);
  float slope2[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = (lane >> 2) + 8 * i;
    slope2[i] = (p.slopes != nullptr && r < live ? p.slopes[head0 + r] : 0.f) * LOG2E;
  }
  pdl_wait();
  const int item = blockIdx.x;
  const int seg = p.decode_seg != nullptr ? p.decode_seg[item] : item;
  const int row = p.seg_q_start[seg], pos = p.seg_pos0[seg];
  const int* table = p.block_table + (size_t)p.seg_slot[seg] * p.table_width;
  const int lowest = lowest_visible(p, pos);
  const int first_tile = lowest / DEC_KEYS, tile_count = pos / DEC_KEYS - first_tile + 1;
  const int share = max((tile_count + p.splits - 1) / p.splits, DEC_MIN_TILES);
  const int begin = first_tile + blockIdx.z * share, end = min(begin + share, first_tile + tile_count);      // exclusive
  const bf16* fresh = p.fresh != nullptr ? p.fresh + (size_t)row * p.fresh_stride + kv_head * D : nullptr;

  for (int idx = threadIdx.x; idx < DEC_ROWS * PIECES; idx += ATTN_THREADS) {
    const int r = idx / PIECES, c = idx - r * PIECES;
    const bool valid = r < live;
    cp_async_16(q_tile + r * PITCH + c * 8, valid ? p.q + (size_t)row * p.q_stride + (head0 + r) * D + c * 8 : p.q, valid);
  }
  // the place of key (tile, lane): looked up a tile ahead of its copies; -2: the new token's own key
  auto look_up = [&](int tile) {
    const int key = tile * DEC_KEYS + lane;
    if (tile >= end || key < lowest || key > pos) return -1;
    if (key == pos && fresh != nullptr) return -2;
    return pool_row(p, table, key, kv_head);
  };
  auto fetch = [&](int place, int stage) {
    bf16* tile = ring + stage * KINDS * TILE;
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i) {
      const int idx = i * 32 + lane, r = idx / PIECES, c = idx - r * PIECES;
      const int at = __shfl_sync(0xffffffffu, place, r);
      const bf16* src = at >= 0 ? p.pool + (size_t)at * D + c * 8 : at == -2 ? fresh + c * 8 : p.pool;
      cp_async_16(tile + r * PITCH + c * 8, src, at != -1);
      if (OWN) cp_async_16(tile + TILE + r * PITCH + c * 8, at >= 0 ? p.values + (size_t)at * D + c * 8 : p.values, at >= 0);
    }
    cp_async_commit();
  };
  int tile = begin + warp;
  int place = look_up(tile), next_place = look_up(tile + ATTN_WARPS);
  fetch(place, 0);                                   // with the queries: one group
  if (fresh != nullptr && block == 0 && pos / DEC_KEYS >= begin && pos / DEC_KEYS < end) {
    const long long slot = p.slots[row];
    if (slot >= 0) {
      const long long page = slot / p.page_size;
      bf16* dst = p.pool + ((page * p.kv_heads + kv_head) * p.page_size + (slot - page * p.page_size)) * D;
      for (int c = threadIdx.x; c < PIECES; c += ATTN_THREADS)
        *reinterpret_cast<uint4*>(dst + c * 8) = __ldcg(reinterpret_cast<const uint4*>(fresh + c * 8));
    }
  }

  const int position[2] = {pos, pos}, limit_lo[2] = {lowest, lowest};
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float o[D / 8][4];
#pragma unroll
  for (int t = 0; t < D / 8; ++t) o[t][0] = o[t][1] = o[t][2] = o[t][3] = 0.f;
  uint32_t q_frag[D / 16][4];
  cp_async_wait<0>();
  __syncthreads();                                   // every thread's pieces of the queries are there
#pragma unroll
  for (int ks = 0; ks < D / 16; ++ks)
    ldmatrix_x4(q_frag[ks], q_tile + ((lane & 7) + (((lane >> 3) & 1) << 3)) * PITCH + (ks * 2 + (lane >> 4)) * 8);
  int stage = 0;
  for (; tile < end; tile += ATTN_WARPS, stage = STAGES == 2 ? stage ^ 1 : 0) {
    if (STAGES == 2 && tile + ATTN_WARPS < end) {
      fetch(next_place, stage ^ 1);
      next_place = look_up(tile + 2 * ATTN_WARPS);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncwarp();
    const bf16* keys = ring + stage * KINDS * TILE;
    float s[DEC_KEYS / 8][4];
    padded_qk<D, DEC_KEYS / 8>(s, q_frag, keys, lane);
    const int key0 = tile * DEC_KEYS;
    if (key0 >= lowest && key0 + DEC_KEYS - 1 <= pos)
      shaped_softmax_step<DEC_KEYS / 8, D / 8, false>(s, o, m, l, key0, position, limit_lo, slope2, p, lane);
    else
      shaped_softmax_step<DEC_KEYS / 8, D / 8, true>(s, o, m, l, key0, position, limit_lo, slope2, p, lane);
    padded_pv<D, DEC_KEYS / 8>(o, s, keys + (KINDS - 1) * TILE, lane);
    __syncwarp();                                    // the next copies go into this tile
    if (STAGES == 1 && tile + ATTN_WARPS < end) {
      fetch(next_place, 0);
      next_place = look_up(tile + 2 * ATTN_WARPS);
    }
  }

  // the warps' parts, in the order of the warps
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = (lane >> 2) + 8 * i;
    if ((lane & 3) == 0) {
      warp_max_[warp][r] = m[i];
      warp_sum_[warp][r] = l[i];
    }
    float* dst = merged + (warp * DEC_ROWS + r) * D + (lane & 3) * 2;
#pragma unroll
    for (int t = 0; t < D / 8; ++t) *reinterpret_cast<float2*>(dst + t * 8) = make_float2(o[t][2 * i], o[t][2 * i + 1]);
  }
  __syncthreads();
  auto finish = [&](float value, float top, float total, int head, int d) {
    float factor = 1.f / total;
    if (p.sinks != nullptr) {
      const float sink = p.sinks[head] * LOG2E, high = fmaxf(top, sink), part = exp2_approx(top - high);
      factor = part / fmaf(total, part, exp2_approx(sink - high));
    }
    value *= factor;
    if (p.gate != nullptr) {
      const unsigned short raw = __ldcg(reinterpret_cast<const unsigned short*>(p.gate + (size_t)row * p.gate_stride + head * D + d));
      value = value / (1.f + expf(-__bfloat162float(*reinterpret_cast<const bf16*>(&raw))));
    }
    p.out[(size_t)row * p.heads * D + head * D + d] = __float2bfloat16_rn(value);
  };
  for (int idx = threadIdx.x; idx < live * D; idx += ATTN_THREADS) {
    const int r = idx / D, d = idx - r * D;
    float top = -INFINITY;
#pragma unroll
    for (int w = 0; w < ATTN_WARPS; ++w) top = fmaxf(top, warp_max_[w][r]);
    float value = 0.f, total = 0.f;
#pragma unroll
    for (int w = 0; w < ATTN_WARPS; ++w) {
      const float part = warp_max_[w][r] == -INFINITY ? 0.f : exp2_approx(warp_max_[w][r] - top);
      value = fmaf(merged[(w * DEC_ROWS + r) * D + d], part, value);
      total = fmaf(warp_sum_[w][r], part, total);
    }
    if (p.splits == 1) {
      finish(value, top, total, head0 + r, d);
    } else {
      const size_t part = ((size_t)item * p.splits + blockIdx.z) * p.heads + head0 + r;
      p.partial[part * D + d] = value;
      if (d == 0) p.limits[part] = make_float2(top, total);
    }
  }
  if (p.splits == 1) return;

  // the last CTA of this (item, heads) to get here adds the parts up, in the order of the keys
  __threadfence();
  __syncthreads();
  int* counter = p.counters + (size_t)item * gridDim.y + blockIdx.y;
  if (threadIdx.x == 0) is_last = atomicAdd(counter, 1) == p.splits - 1;
  __syncthreads();
  if (!is_last) return;
  __threadfence();
  if (threadIdx.x == 0) *counter = 0;
  // a factor per (head, part): the parts' maxima brought together, a warp per head, lanes over the parts
  float* factors = merged;                                   // [16][splits]
  const size_t first_part = (size_t)item * p.splits * p.heads + head0;
  for (int r = warp; r < live; r += ATTN_WARPS) {
    float2 mine[DEC_MAX_SPLITS / 32];
    float top = -INFINITY;
#pragma unroll
    for (int k = 0; k < DEC_MAX_SPLITS / 32; ++k) {
      const int z = k * 32 + lane;
      mine[k] = z < p.splits ? __ldcg(&p.limits[first_part + (size_t)z * p.heads + r]) : make_float2(-INFINITY, 0.f);
      top = fmaxf(top, mine[k].x);
    }
    top = warp_max(top);
    float total = 0.f;
#pragma unroll
    for (int k = 0; k < DEC_MAX_SPLITS / 32; ++k) {
      const float part = mine[k].x == -INFINITY ? 0.f : exp2_approx(mine[k].x - top);
      if (k * 32 + lane < p.splits) factors[r * p.splits + k * 32 + lane] = part;
      total = fmaf(mine[k].y, part, total);
    }
    total = warp_sum(total);
    if (lane == 0) {
      warp_max_[0][r] = top;
      warp_sum_[0][r] = total;
    }
  }
  __syncthreads();
  for (int idx = threadIdx.x * 4; idx < live * D; idx += ATTN_THREADS * 4) {
    const int r = idx / D, d = idx - r * D;
    const float* src = p.partial + (first_part + r) * D + d;
    const size_t step = (size_t)p.heads * D;
    float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int z = 0; z < p.splits; ++z) {
      const float4 v = __ldcg(reinterpret_cast<const float4*>(src + z * step));
      const float part = factors[r * p.splits + z];
      sum.x = fmaf(v.x, part, sum.x); sum.y = fmaf(v.y, part, sum.y);
      sum.z = fmaf(v.z, part, sum.z); sum.w = fmaf(v.w, part, sum.w);
    }
    finish(sum.x, warp_max_[0][r], warp_sum_[0][r], head0 + r, d);
    finish(sum.y, warp_max_[0][r], warp_sum_[0][r], head0 + r, d + 1);
    finish(sum.z, warp_max_[0][r], warp_sum_[0][r], head0 + r, d + 2);
    finish(sum.w, warp_max_[0][r], warp_sum_[0][r], head0 + r, d + 3);
  }
}

template <int D, bool OWN>
static int launch_shaped_prefill(const ShapedArgs& p, int tiles, cudaStream_t stream) {
  const size_t shared = sizeof(bf16) * (size_t)(TILE_Q + (OWN ? 4 : 2) * TILE_KV) * (D + 8);
  if (shared > 48 * 1024) {
    cudaError_t err = cudaFuncSetAttribute(shaped_prefill_kernel<D, OWN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared);
    if (err != cudaSuccess) return (int)err;
  }
  launch_kernel(shaped_prefill_kernel<D, OWN>, dim3(tiles, p.heads), dim3(ATTN_THREADS), shared, stream, p);
  return launch_status();
}

template <int D, bool OWN>
static int launch_shaped_decode(const ShapedArgs& p, int items, cudaStream_t stream) {
  const size_t tiles = sizeof(bf16) * (size_t)ATTN_WARPS * DEC_STAGES<D, OWN> * (OWN ? 2 : 1) * DEC_KEYS * (D + 8);
  const size_t parts = sizeof(float) * (size_t)ATTN_WARPS * DEC_ROWS * D;
  const size_t shared = sizeof(bf16) * (size_t)DEC_ROWS * (D + 8) + (tiles > parts ? tiles : parts);
  if (shared > 48 * 1024) {
    cudaError_t err = cudaFuncSetAttribute(shaped_decode_kernel<D, OWN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared);
    if (err != cudaSuccess) return (int)err;
  }
  const int per = p.heads / p.kv_heads;
  launch_kernel(shaped_decode_kernel<D, OWN>, dim3(items, p.kv_heads * ((per + DEC_ROWS - 1) / DEC_ROWS), p.splits),
                dim3(ATTN_THREADS), shared, stream, p);
  return launch_status();
}

template <int D>
static int launch_shaped(const ShapedArgs& p, int decode, int count, cudaStream_t stream) {
  if (p.values != nullptr)
    return decode ? launch_shaped_decode<D, true>(p, count, stream) : launch_shaped_prefill<D, true>(p, count, stream);
  return decode ? launch_shaped_decode<D, false>(p, count, stream) : launch_shaped_prefill<D, false>(p, count, stream);
}

}  // namespace mlr

using namespace mlr;

MLR_DEFINE_PDL_SWITCH

// Whether the kernels take this head size.
MLR_EXPORT int mlr_attention_shaped_mma_fits(int dim) { return dim == 32 || dim == 64 || dim == 96 || dim == 128; }

// decode == 0: tiles of up to 64 rows of one segment (list_a: segments, list_b: first rows; `count` of them).
// decode == 1: `count` one-row segments (list_a: the segments, or null: segments 0 .. count - 1), keys cut over
// `splits` CTAs; partial: float32 [count, splits, heads, dim + 2] and counters: `count` * kv_heads * blocks of 16
// heads zeros (left zero), both only with splits > 1.
// q, gate, fresh: bfloat16 rows with strides (in elements); gate null: no gate; fresh null: the new keys are in
// the pool already, else `slots` (int64 per row) says where they go (only where keys are the values: values null; else
// values [pages, kv_heads, page_size, dim]).  softcap 0: no cap; slopes, sinks: float32
// [heads] or null; chunk, window 0: none.
MLR_EXPORT int mlr_attention_shaped_mma(int decode, const void* q, long long q_stride, const void* fresh,
                                        long long fresh_stride, const long long* slots, void* pool, const void* values,
                                        void* out, const void* gate, long long gate_stride, const float* slopes, const float* sinks,
                                        const int* list_a, const int* list_b, int count, const int* seg_q_start,
                                        const int* seg_q_len, const int* seg_pos0, const int* block_table,
                                        const int* seg_slot, int table_width, int heads, int kv_heads, int dim,
                                        int page_size, int window, int chunk, float scale, float softcap, float* partial,
                                        int* counters, int splits, cudaStream_t stream) {
  if (count == 0) return MLR_OK;
  if (count < 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || page_size <= 0 || table_width <= 0 ||
      window < 0 || chunk < 0 || softcap < 0.f || splits < 1 || (fresh != nullptr && (slots == nullptr || values != nullptr)) ||
      (splits > 1 && (partial == nullptr || counters == nullptr)))
    return MLR_BAD_SIZE;
  auto aligned = [](const void* ptr) { return (reinterpret_cast<uintptr_t>(ptr) & 15) == 0; };
  if (!aligned(q) || !aligned(fresh) || !aligned(pool) || !aligned(values) || !aligned(out) || q_stride % 8 || fresh_stride % 8 ||
      gate_stride % 2 || (reinterpret_cast<uintptr_t>(gate) & 3))
    return MLR_BAD_ALIGNMENT;
  if (heads > 65535 || splits > DEC_MAX_SPLITS) return MLR_TOO_LARGE;
  ShapedArgs p;
  p.q = (const bf16*)q; p.q_stride = q_stride;
  p.fresh = (const bf16*)fresh; p.fresh_stride = fresh_stride; p.slots = slots;
  p.pool = (bf16*)pool; p.values = (const bf16*)values; p.out = (bf16*)out; p.gate = (const bf16*)gate; p.gate_stride = gate_stride;
  p.slopes = slopes; p.sinks = sinks;
  p.tile_seg = list_a; p.tile_row0 = list_b; p.decode_seg = list_a;
  p.seg_q_start = seg_q_start; p.seg_q_len = seg_q_len; p.seg_pos0 = seg_pos0;
  p.block_table = block_table; p.seg_slot = seg_slot; p.table_width = table_width;
  p.heads = heads; p.kv_heads = kv_heads; p.page_size = page_size;
  p.page_shift = -1;
  for (int s = 0; s < 20; ++s)
    if ((1 << s) == page_size) p.page_shift = s;
  p.window = window; p.chunk = chunk;
  p.capped = softcap > 0.f;
  p.in_scale = p.capped ? scale / softcap : scale * LOG2E;
  p.out_scale = p.capped ? softcap * LOG2E : 1.f;
  p.partial = partial;                             // the parts, then their maxima and denominators
  p.limits = partial == nullptr ? nullptr : reinterpret_cast<float2*>(partial + (size_t)count * splits * heads * dim);
  p.counters = counters; p.splits = splits;
  switch (dim) {
    case 32: return launch_shaped<32>(p, decode, count, stream);
    case 64: return launch_shaped<64>(p, decode, count, stream);
    case 96: return launch_shaped<96>(p, decode, count, stream);
    case 128: return launch_shaped<128>(p, decode, count, stream);
    default: return MLR_BAD_SIZE;
  }
}
