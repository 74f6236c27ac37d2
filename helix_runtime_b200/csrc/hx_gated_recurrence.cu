// A real-gated linear recurrence per channel, with gates from block-diagonal matrices: what runs
// between the matrix products of such a mixer.
//
//   r_t = sigmoid(R_b u_t + br),  i_t = sigmoid(I_b u_t + bi)        (block b of the channels)
//   log a_t = -rate * r_t,  S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t,  out_t = S_t f(y_t + by)
//
// with u the filtered branch, y the other branch, f = gelu_tanh and `rate` one positive number per
// channel.  The state S is float32, one number per channel and request, zero at admission.
//
// A decay close to one loses its digits in float32, so it is carried as d = a - 1 = expm1(log a)
// everywhere: 1 - a^2 = -d (2 + d), a step is S + (d S + push), and two stretches of time with
// (d1, p1), (d2, p2) join to (d1 + d2 + d1 d2, p1 + d2 p1 + p2).
//
// Forms.
//   * Any sizes, both dtypes: hx_block_gates computes d and push = sqrt(1 - a^2) i u for every
//     token and channel with CUDA-core products (tiles of 64 tokens x 64 channels, both gates
//     of a channel in one thread, so the gate arithmetic is the product's epilogue), and
//     hx_gated_scan walks token by token, one thread per channel, carrying the rounding of every
//     step beside the state, so that the error does not grow with the position.
//   * bfloat16, blocks of a multiple of 8 channels: hx_block_gates_tiled and hx_gated_scan_tiled cut
//     time into tiles of 64 tokens that all run at once.  The gates' products run on mma.sync:
//     a block is so small (a few hundred reduction steps) that the arithmetic behind the sums
//     decides the time, and here every warp of the SM does it, straight from its accumulators.
//   * hx_gated_recurrence_step (bfloat16, one token per request): gates, update and output in
//     one kernel.  A CTA owns 16 channels and streams their 32 gate rows once for all tokens
//     of the step, as 16-row operands of mma.sync straight from global memory (the order of
//     the reduction is free, so every lane loads whole 16-byte pieces), its four warps cutting
//     the reduction.
#include "hx_mma.cuh"

namespace {

// sqrt(1 - a^2) i u from d = a - 1
__device__ __forceinline__ float push_of(float d, float i, float u) {
  return sqrtf(-d * (2.0f + d)) * i * u;
}

// ------------------------------------------------------------------ gates, any sizes

constexpr int GATE_TILE = 64;
constexpr int GATE_DEPTH = 16;

template <typename T>
struct GateArgs {
  const T* u;                // [tokens, ld_u]
  int ld_u;
  const T* w;                // [blocks][2][size][size]: the rows of R, then of I
  const float* r_bias;       // [blocks * size]
  const float* i_bias;
  const float* rate;
  float* decay;              // [tokens, channels]: d
  float* push;               // [tokens, channels]
  int tokens, size, channels;
};

template <typename T>
__global__ __launch_bounds__(256) void block_gates_kernel(const GateArgs<T> a) {
  __shared__ float us[GATE_DEPTH][GATE_TILE + 4];
  __shared__ float rs[GATE_DEPTH][GATE_TILE + 4];
  __shared__ float is[GATE_DEPTH][GATE_TILE + 4];
  hx_pdl_prologue();
  const int block = blockIdx.z;
  const int token0 = blockIdx.x * GATE_TILE;
  const int out0 = blockIdx.y * GATE_TILE;
  const int size = a.size;
  const T* u = a.u + static_cast<size_t>(block) * size;
  const T* wr = a.w + static_cast<size_t>(block) * 2 * size * size;
  const T* wi = wr + static_cast<size_t>(size) * size;
  const int tx = threadIdx.x & 15;
  const int ty = threadIdx.x >> 4;
  float r_sum[4][4], i_sum[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) r_sum[i][j] = i_sum[i][j] = 0.0f;
  for (int k0 = 0; k0 < size; k0 += GATE_DEPTH) {
    __syncthreads();
    for (int e = threadIdx.x; e < GATE_TILE * GATE_DEPTH; e += 256) {
      const int row = e / GATE_DEPTH, k = e - row * GATE_DEPTH;
      const int token = token0 + row, o = out0 + row, i = k0 + k;
      us[k][row] = (token < a.tokens && i < size)
                       ? hx_to_float<T>(u[static_cast<size_t>(token) * a.ld_u + i]) : 0.0f;
      const bool there = o < size && i < size;
      rs[k][row] = there ? hx_to_float<T>(wr[static_cast<size_t>(o) * size + i]) : 0.0f;
      is[k][row] = there ? hx_to_float<T>(wi[static_cast<size_t>(o) * size + i]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < GATE_DEPTH; ++k) {
      const float4 x = *reinterpret_cast<const float4*>(&us[k][ty * 4]);
      const float4 p = *reinterpret_cast<const float4*>(&rs[k][tx * 4]);
      const float4 q = *reinterpret_cast<const float4*>(&is[k][tx * 4]);
      const float xv[4] = {x.x, x.y, x.z, x.w};
      const float pv[4] = {p.x, p.y, p.z, p.w};
      const float qv[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          r_sum[i][j] = fmaf(xv[i], pv[j], r_sum[i][j]);
          i_sum[i][j] = fmaf(xv[i], qv[j], i_sum[i][j]);
        }
    }
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int o = out0 + tx * 4 + j;
    if (o >= size) continue;
    const int c = block * size + o;
    const float br = a.r_bias[c], bi = a.i_bias[c], rate = a.rate[c];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int token = token0 + ty * 4 + i;
      if (token >= a.tokens) continue;
      const float d = expm1f(-rate * hx_sigmoid(r_sum[i][j] + br));
      const float x = hx_to_float<T>(u[static_cast<size_t>(token) * a.ld_u + o]);
      const size_t index = static_cast<size_t>(token) * a.channels + c;
      a.decay[index] = d;
      a.push[index] = push_of(d, hx_sigmoid(i_sum[i][j] + bi), x);
    }
  }
}

// ------------------------------------------------------------------------ the scan

template <typename T>
struct GatedScanArgs {
  const float* decay;        // [tokens, channels]
  const float* push;
  const T* y;                // [tokens, ld_y], or null: taken from `accum`
  int ld_y;
  float* accum;              // [tokens, ld_accum] float32 sums, y's columns first; cleared here,
  int ld_accum;              // the `accum_columns` columns of every row
  const float* y_bias;       // [channels]
  float* state;              // per slot: [channels]
  long long state_stride;
  T* out;                    // [tokens, ld_out]
  int ld_out;
  int channels;
  const int* request_start;
  const int* request_slot;
};

// the other branch's value of (token, c), rounded as the projection's own store rounds it
template <typename T>
__device__ __forceinline__ float other_branch(const T* y, int ld_y, const float* accum, int ld_accum,
                                              int token, int c) {
  if (y != nullptr) return hx_to_float<T>(y[static_cast<size_t>(token) * ld_y + c]);
  return hx_to_float<T>(hx_from_float<T>(accum[static_cast<size_t>(token) * ld_accum + c]));
}

// the sums of both branches at (token, c) have been read: clear them
__device__ __forceinline__ void clear_sums(float* accum, int ld_accum, int channels, int token, int c) {
  float* row = accum + static_cast<size_t>(token) * ld_accum;
  row[c] = 0.0f;
  row[channels + c] = 0.0f;
}

// One thread per channel, token by token.  What a step's rounding loses (a
// two-sum recovers it) is carried beside the state and decays like it.
template <typename T>
__global__ __launch_bounds__(64) void gated_scan_kernel(const GatedScanArgs<T> a) {
  hx_pdl_prologue();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= a.channels) return;
  const int request = blockIdx.y;
  const int start = a.request_start[request];
  const int count = a.request_start[request + 1] - start;
  if (count <= 0) return;
  float* state = a.state + static_cast<size_t>(a.request_slot[request]) * a.state_stride;
  float S = state[c], carry = 0.0f;
  const float bias = a.y_bias[c];
  for (int t = start; t < start + count; ++t) {
    const size_t index = static_cast<size_t>(t) * a.channels + c;
    const float d = a.decay[index];
    const float add = fmaf(d, S, a.push[index]);
    const float sum = S + add;
    const float shadow = sum - S;
    const float error = (S - (sum - shadow)) + (add - shadow);
    carry = fmaf(d, carry, carry) + error;
    S = sum;
    const float y = other_branch(a.y, a.ld_y, a.accum, a.ld_accum, t, c);
    a.out[static_cast<size_t>(t) * a.ld_out + c] =
        hx_from_float<T>((S + carry) * hx_gelu_tanh(y + bias));
    if (a.y == nullptr) clear_sums(a.accum, a.ld_accum, a.channels, t, c);
  }
  state[c] = S + carry;
}

// ------------------------------------------------------- gates and scan by tiles of 64 tokens
//
// Time is cut into tiles of 64 tokens, counted from each request's first token of the step
// (numbered over the batch as hx_find_query_tile numbers them).  The gates' kernel leaves, beside
// decay and push, every tile's composition (d, p): the tile takes a state S to S + (d S + p).  The
// scan's kernel composes the tiles in front of its own, starts from the state as it was before
// the step (`before`, copied by the gates' kernel: the tile that writes the new state does not
// wait for the others to have read the old one) and runs its 64 tokens.

constexpr int TILE_TOKENS = 64;
constexpr int TILE_WARPS = 8;
constexpr int TILE_CHANNELS = TILE_WARPS * 16;      // of the gates' kernel: a warp has 16
constexpr int TILE_DEPTH = 256;                     // reduction steps staged at once
constexpr int TILE_STRIDE = TILE_DEPTH + 32;        // row stride: two rows fall on all 32 banks

struct Joined {
  float d, p;
};
__device__ __forceinline__ Joined then(const Joined& first, const Joined& second) {
  return {first.d + fmaf(second.d, first.d, second.d), first.p + fmaf(second.d, first.p, second.p)};
}

// exp(x) - 1 for x <= 0: seven terms of the series near zero (remainder below 2e-8 of the result),
// the hardware exponential elsewhere, where the difference keeps its digits.
__device__ __forceinline__ float fast_expm1(float x) {
  float series = fmaf(x, 1.0f / 7.0f, 1.0f);
  series = fmaf(series * x, 1.0f / 6.0f, 1.0f);
  series = fmaf(series * x, 1.0f / 5.0f, 1.0f);
  series = fmaf(series * x, 1.0f / 4.0f, 1.0f);
  series = fmaf(series * x, 1.0f / 3.0f, 1.0f);
  series = fmaf(series * x, 1.0f / 2.0f, 1.0f);
  return x > -0.35f ? series * x : __expf(x) - 1.0f;
}

__device__ __forceinline__ float fast_sqrt(float x) {
  float y;
  asm("sqrt.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// decay and push of one (token, channel) from the gates' sums, with the hardware functions.  Both
// sigmoids share one reciprocal, 1 / ((1 + e^-r)(1 + e^-i)); sums below -43 (a gate of 2e-19) are
// taken as -43 so that the product stays a number.
__device__ __forceinline__ Joined fast_gates(float r_sum, float i_sum, float rate, float u) {
  const float r = 1.0f + __expf(-fmaxf(r_sum, -43.0f));
  const float i = 1.0f + __expf(-fmaxf(i_sum, -43.0f));
  const float both = __fdividef(1.0f, r * i);
  const float d = fast_expm1(-rate * (both * i));
  return {d, fast_sqrt(-d * (2.0f + d)) * (both * r) * u};
}

struct TiledGateArgs {
  const __nv_bfloat16* u;    // [tokens, ld_u]
  int ld_u;
  const __nv_bfloat16* w;    // [blocks][2][size][size]
  const float* r_bias;
  const float* i_bias;
  const float* rate;
  float* decay;              // [tokens, channels]
  float* push;
  float2* joined;            // [tiles, channels]
  const float* state;        // per slot: [channels]
  long long state_stride;
  float* before;             // [requests, channels]
  const int* request_start;
  const int* request_slot;
  int requests, size, channels;
  int channel_tiles;         // of a block
};

__global__ __launch_bounds__(TILE_WARPS * 32, 2) void tiled_gates_kernel(const TiledGateArgs a) {
  __shared__ __align__(16) __nv_bfloat16 us[TILE_TOKENS][TILE_STRIDE];
  hx_pdl_trigger();
  const int warp = threadIdx.x >> 5;
  const int lane = threadIdx.x & 31;
  const int group = lane >> 2, quad = lane & 3;
  int tile = 0, tiles = 0;
  const int request = hx_find_query_tile(a.request_start, a.requests, 1, TILE_TOKENS, blockIdx.y,
                                         tile, tiles);
  if (request < 0) {
    hx_pdl_wait();      // a grid must not be seen complete before its predecessor is
    return;
  }
  const int first = a.request_start[request] + tile * TILE_TOKENS;
  const int here = min(TILE_TOKENS, a.request_start[request + 1] - first);
  const int size = a.size;
  const int block = blockIdx.x / a.channel_tiles;
  const int tile0 = (blockIdx.x - block * a.channel_tiles) * TILE_CHANNELS;
  const int out0 = tile0 + warp * 16;
  const int pieces = size / 8;
  const bool busy = out0 < size;      // the whole warp
  const __nv_bfloat16* wr = a.w + static_cast<size_t>(block) * 2 * size * size;
  const __nv_bfloat16* wi = wr + static_cast<size_t>(size) * size;
  const int row_lo = min(out0 + group, size - 1);      // rows behind the block are not used
  const int row_hi = min(out0 + group + 8, size - 1);
  auto weight = [&](const __nv_bfloat16* w, int row, int piece) {
    return busy && piece < pieces
               ? __ldg(reinterpret_cast<const uint4*>(w + static_cast<size_t>(row) * size) + piece)
               : make_uint4(0u, 0u, 0u, 0u);
  };
  // a turn is 32 reduction steps: a lane holds one 16-byte piece of its two rows of each matrix
  const int turns = (pieces + 3) / 4;
  uint4 next[4];      // the turn after the one that is worked on
  auto fetch = [&](int turn) {
    const int piece = turn * 4 + quad;
    next[0] = weight(wr, row_lo, piece);
    next[1] = weight(wr, row_hi, piece);
    next[2] = weight(wi, row_lo, piece);
    next[3] = weight(wi, row_hi, piece);
  };
  fetch(0);
  hx_pdl_wait();
  // columns [column0, column0 + count) of the block's part of u, `count` a multiple of 8
  auto stage = [&](int column0, int count) {
    // a warp takes every eighth token, a lane one 16-byte piece; all loads in flight together
    uint4 x[TILE_TOKENS / TILE_WARPS];
#pragma unroll
    for (int t = 0; t < TILE_TOKENS / TILE_WARPS; ++t) {
      const int token = warp + t * TILE_WARPS;
      x[t] = make_uint4(0u, 0u, 0u, 0u);
      if (token < here && lane * 8 < count)
        x[t] = *(reinterpret_cast<const uint4*>(a.u + static_cast<size_t>(first + token) * a.ld_u +
                                                static_cast<size_t>(block) * size + column0) + lane);
    }
#pragma unroll
    for (int t = 0; t < TILE_TOKENS / TILE_WARPS; ++t)
      if (lane * 8 < count) *reinterpret_cast<uint4*>(&us[warp + t * TILE_WARPS][lane * 8]) = x[t];
  };
  float r[8][4], i[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) r[n][e] = i[n][e] = 0.0f;
  for (int k0 = 0; k0 < size; k0 += TILE_DEPTH) {
    const int depth = min(TILE_DEPTH, size - k0);
    if (k0 > 0) __syncthreads();
    stage(k0, depth);
    __syncthreads();
    if (!busy) continue;
    const int last = (depth + 31) / 32;
    for (int t = 0; t < last; ++t) {
      const uint4 r_lo = next[0], r_hi = next[1], i_lo = next[2], i_hi = next[3];
      if (k0 / 32 + t + 1 < turns) fetch(k0 / 32 + t + 1);
      const bool there = t * 32 + quad * 8 < depth;      // a piece behind the rows is stale
      const uint32_t r_first[4] = {r_lo.x, r_hi.x, r_lo.y, r_hi.y};
      const uint32_t r_second[4] = {r_lo.z, r_hi.z, r_lo.w, r_hi.w};
      const uint32_t i_first[4] = {i_lo.x, i_hi.x, i_lo.y, i_hi.y};
      const uint32_t i_second[4] = {i_lo.z, i_hi.z, i_lo.w, i_hi.w};
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        uint4 x = *reinterpret_cast<const uint4*>(&us[n * 8 + group][t * 32 + quad * 8]);
        if (!there) x = make_uint4(0u, 0u, 0u, 0u);
        hx_mma_bf16(r[n], r_first, x.x, x.y);
        hx_mma_bf16(r[n], r_second, x.z, x.w);
        hx_mma_bf16(i[n], i_first, x.x, x.y);
        hx_mma_bf16(i[n], i_second, x.z, x.w);
      }
    }
  }
  // the tile's own channels of u, for the input gate
  int column0 = tile0;
  if (size > TILE_DEPTH) {
    __syncthreads();
    stage(tile0, min(TILE_CHANNELS, size - tile0));
    __syncthreads();
    column0 = 0;
  }
  if (!busy) return;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int o = out0 + group + half * 8;
    const bool live = o < size;
    const int c = block * size + (live ? o : 0);
    const float br = a.r_bias[c], bi = a.i_bias[c], rate = a.rate[c];
    const int column = column0 + (live ? warp * 16 + group + half * 8 : 0);
    Joined all = {0.0f, 0.0f};
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      Joined pair = {0.0f, 0.0f};
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int token = n * 8 + quad * 2 + e;
        if (token >= here) continue;      // a token that is not there changes nothing
        const Joined one = fast_gates(r[n][half * 2 + e] + br, i[n][half * 2 + e] + bi, rate,
                                      __bfloat162float(us[token][column]));
        if (live) {
          const size_t index = static_cast<size_t>(first + token) * a.channels + c;
          a.decay[index] = one.d;
          a.push[index] = one.p;
        }
        pair = then(pair, one);
      }
      // the eight tokens' pairs sit in the four lanes of a quad, in order
#pragma unroll
      for (int step = 1; step < 4; step *= 2) {
        const Joined other = {__shfl_xor_sync(0xffffffffu, pair.d, step),
                              __shfl_xor_sync(0xffffffffu, pair.p, step)};
        pair = (quad & step) ? then(other, pair) : then(pair, other);
      }
      all = then(all, pair);
    }
    if (live && quad == 0) {
      a.joined[static_cast<size_t>(blockIdx.y) * a.channels + c] = make_float2(all.d, all.p);
      if (tile == 0)
        a.before[static_cast<size_t>(request) * a.channels + c] =
            a.state[static_cast<size_t>(a.request_slot[request]) * a.state_stride + c];
    }
  }
}

constexpr int SCAN_CHANNELS = 32;      // per CTA: one warp's lanes
constexpr int SCAN_WARPS = 8;
constexpr int SCAN_RUN = TILE_TOKENS / SCAN_WARPS;      // tokens of a warp

struct TiledScanArgs {
  GatedScanArgs<__nv_bfloat16> scan;
  const float2* joined;
  const float* before;
  int requests;
};

__global__ __launch_bounds__(SCAN_WARPS * 32) void tiled_scan_kernel(const TiledScanArgs args) {
  __shared__ Joined shared[2][SCAN_WARPS][SCAN_CHANNELS];
  hx_pdl_trigger();
  const GatedScanArgs<__nv_bfloat16>& a = args.scan;
  const int lane = threadIdx.x & 31;
  const int warp = threadIdx.x >> 5;
  const int c = blockIdx.x * SCAN_CHANNELS + lane;
  const bool live = c < a.channels;
  int tile = 0, tiles = 0;
  const int request = hx_find_query_tile(a.request_start, args.requests, 1, TILE_TOKENS, blockIdx.y,
                                         tile, tiles);
  hx_pdl_wait();
  if (request < 0) return;      // the whole CTA
  const int start = a.request_start[request] + tile * TILE_TOKENS + warp * SCAN_RUN;
  const int here = a.request_start[request + 1] - start;      // tokens from this warp's first on
  Joined step[SCAN_RUN];
  float y[SCAN_RUN];
#pragma unroll
  for (int k = 0; k < SCAN_RUN; ++k) {
    const bool there = live && k < here;
    const size_t index = static_cast<size_t>(start + k) * a.channels + c;
    step[k].d = there ? a.decay[index] : 0.0f;      // a token that is not there changes nothing
    step[k].p = there ? a.push[index] : 0.0f;
    y[k] = there ? other_branch(a.y, a.ld_y, a.accum, a.ld_accum, start + k, c) : 0.0f;
  }
  const float bias = live ? a.y_bias[c] : 0.0f;
  float S = live ? args.before[static_cast<size_t>(request) * a.channels + c] : 0.0f;
  // the tiles in front of this one, an equal run of them per warp
  const int run = (tile + SCAN_WARPS - 1) / SCAN_WARPS;
  Joined front = {0.0f, 0.0f};
  const float2* earlier = args.joined + static_cast<size_t>(blockIdx.y - tile) * a.channels + c;
  const int end = min((warp + 1) * run, tile);
#pragma unroll 4
  for (int t = warp * run; t < end; ++t) {
    const float2 j = live ? earlier[static_cast<size_t>(t) * a.channels] : make_float2(0.0f, 0.0f);
    front = then(front, Joined{j.x, j.y});
  }
  Joined own = {0.0f, 0.0f};
#pragma unroll
  for (int k = 0; k < SCAN_RUN; ++k) own = then(own, step[k]);
  shared[0][warp][lane] = front;
  shared[1][warp][lane] = own;
  __syncthreads();
#pragma unroll
  for (int w = 0; w < SCAN_WARPS; ++w) {
    const Joined j = shared[0][w][lane];
    S = S + fmaf(j.d, S, j.p);
  }
#pragma unroll
  for (int w = 0; w < SCAN_WARPS; ++w) {
    const Joined j = shared[1][w][lane];
    if (w < warp) S = S + fmaf(j.d, S, j.p);
  }
  if (!live) return;
#pragma unroll
  for (int k = 0; k < SCAN_RUN; ++k) {
    S = S + fmaf(step[k].d, S, step[k].p);
    if (k < here) {
      a.out[static_cast<size_t>(start + k) * a.ld_out + c] =
          __float2bfloat16_rn(S * hx_gelu_tanh_fast(y[k] + bias));
      if (a.y == nullptr) clear_sums(a.accum, a.ld_accum, a.channels, start + k, c);
    }
  }
  // the warp that ran the last token knows the new state (the ones behind it changed nothing)
  if (tile == tiles - 1 && warp == SCAN_WARPS - 1)
    a.state[static_cast<size_t>(a.request_slot[request]) * a.state_stride + c] = S;
}

// --------------------------------------------------- one token per request, all in one

constexpr int STEP_WARPS = 4;
constexpr int STEP_CHANNELS = 16;

struct StepArgs {
  const __nv_bfloat16* u;      // [tokens, ld_u]
  int ld_u;
  const __nv_bfloat16* w;      // [blocks][2][size][size]
  const float* r_bias;
  const float* i_bias;
  const float* rate;
  GatedScanArgs<__nv_bfloat16> scan;
  const int* token_request;
  int tokens, size, tiles;     // tiles: 16-channel tiles of a block
};

// GROUPS: groups of eight tokens a CTA works on at a time.
template <int GROUPS>
__global__ __launch_bounds__(STEP_WARPS * 32) void gated_recurrence_step_kernel(const StepArgs a) {
  constexpr int TOKENS = GROUPS * 8;
  __shared__ float sums[STEP_WARPS][2][STEP_CHANNELS][TOKENS + 1];
  hx_pdl_trigger();
  const int warp = threadIdx.x >> 5;
  const int lane = threadIdx.x & 31;
  const int group = lane >> 2, quad = lane & 3;
  const int block = blockIdx.x / a.tiles;
  const int out0 = (blockIdx.x - block * a.tiles) * STEP_CHANNELS;
  const int size = a.size;
  const int pieces = size / 8;
  const __nv_bfloat16* wr = a.w + static_cast<size_t>(block) * 2 * size * size;
  const __nv_bfloat16* wi = wr + static_cast<size_t>(size) * size;
  const int row_lo = min(out0 + group, size - 1);      // rows behind the block are not used
  const int row_hi = min(out0 + group + 8, size - 1);
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  // Four 16-byte pieces (32 reduction steps) at a time, the warps taking turns: the weights of
  // this warp's first turn do not depend on the kernel before and are fetched before the wait.
  auto weight = [&](const __nv_bfloat16* w, int row, int piece) {
    return piece < pieces ? __ldg(reinterpret_cast<const uint4*>(w + static_cast<size_t>(row) * size) + piece)
                          : zero;
  };
  uint4 r_lo, r_hi, i_lo, i_hi;
  auto fetch = [&](int turn) {
    const int piece = turn * 4 + quad;
    r_lo = weight(wr, row_lo, piece);
    r_hi = weight(wr, row_hi, piece);
    i_lo = weight(wi, row_lo, piece);
    i_hi = weight(wi, row_hi, piece);
  };
  const int turns = (pieces + 3) / 4;
  if (warp < turns) fetch(warp);
  // behind the products a thread owns one channel of every eighth token
  constexpr int PER_THREAD = TOKENS * STEP_CHANNELS / (STEP_WARPS * 32);
  constexpr int STEP = STEP_WARPS * 32 / STEP_CHANNELS;
  const int channel = threadIdx.x & (STEP_CHANNELS - 1);
  const int local0 = threadIdx.x / STEP_CHANNELS;
  const int o = out0 + channel;
  const int c = block * size + min(o, size - 1);
  const float br = a.r_bias[c], bi = a.i_bias[c], rate = a.rate[c], by = a.scan.y_bias[c];
  int slots[PER_THREAD];
  auto look_up = [&](int token0) {
#pragma unroll
    for (int k = 0; k < PER_THREAD; ++k) {
      const int token = token0 + local0 + k * STEP;
      slots[k] = token < a.tokens ? a.scan.request_slot[a.token_request[token]] : -1;
    }
  };
  look_up(0);
  hx_pdl_wait();

  for (int token0 = 0; token0 < a.tokens; token0 += TOKENS) {
    if (token0 > 0) look_up(token0);
    // in flight during the products
    float S[PER_THREAD], y[PER_THREAD], u[PER_THREAD];
#pragma unroll
    for (int k = 0; k < PER_THREAD; ++k) {
      const int token = token0 + local0 + k * STEP;
      S[k] = y[k] = u[k] = 0.0f;
      if (slots[k] >= 0) {
        S[k] = a.scan.state[static_cast<size_t>(slots[k]) * a.scan.state_stride + c];
        y[k] = other_branch(a.scan.y, a.scan.ld_y, a.scan.accum, a.scan.ld_accum, token, c);
        u[k] = __bfloat162float(a.u[static_cast<size_t>(token) * a.ld_u + c]);
      }
    }
    float r[GROUPS][4], i[GROUPS][4];
#pragma unroll
    for (int g = 0; g < GROUPS; ++g)
#pragma unroll
      for (int e = 0; e < 4; ++e) r[g][e] = i[g][e] = 0.0f;
    for (int turn = warp; turn < turns; turn += STEP_WARPS) {
      if (token0 > 0 || turn != warp) fetch(turn);
      const int piece = turn * 4 + quad;
      uint4 x[GROUPS];
#pragma unroll
      for (int g = 0; g < GROUPS; ++g) {
        const int token = token0 + g * 8 + group;
        x[g] = token < a.tokens && piece < pieces
                   ? *(reinterpret_cast<const uint4*>(a.u + static_cast<size_t>(token) * a.ld_u +
                                                      static_cast<size_t>(block) * size) + piece)
                   : zero;
      }
      // a lane's eight reduction steps feed two products of sixteen: words 0, 1 the first and
      // words 2, 3 the second (weights and inputs are dealt alike)
      const uint32_t r_first[4] = {r_lo.x, r_hi.x, r_lo.y, r_hi.y};
      const uint32_t r_second[4] = {r_lo.z, r_hi.z, r_lo.w, r_hi.w};
      const uint32_t i_first[4] = {i_lo.x, i_hi.x, i_lo.y, i_hi.y};
      const uint32_t i_second[4] = {i_lo.z, i_hi.z, i_lo.w, i_hi.w};
#pragma unroll
      for (int g = 0; g < GROUPS; ++g) {
        hx_mma_bf16(r[g], r_first, x[g].x, x[g].y);
        hx_mma_bf16(r[g], r_second, x[g].z, x[g].w);
        hx_mma_bf16(i[g], i_first, x[g].x, x[g].y);
        hx_mma_bf16(i[g], i_second, x[g].z, x[g].w);
      }
    }
    if (token0 > 0) __syncthreads();      // the sums of the tokens before have been read
#pragma unroll
    for (int g = 0; g < GROUPS; ++g)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int channel = group + (e >> 1) * 8, token = g * 8 + quad * 2 + (e & 1);
        sums[warp][0][channel][token] = r[g][e];
        sums[warp][1][channel][token] = i[g][e];
      }
    __syncthreads();
    if (o < size) {
#pragma unroll
      for (int k = 0; k < PER_THREAD; ++k) {
        if (slots[k] < 0) continue;
        const int local = local0 + k * STEP, token = token0 + local;
        float r_sum = br, i_sum = bi;
#pragma unroll
        for (int w = 0; w < STEP_WARPS; ++w) {
          r_sum += sums[w][0][channel][local];
          i_sum += sums[w][1][channel][local];
        }
        const Joined one = fast_gates(r_sum, i_sum, rate, u[k]);
        const float state = S[k] + fmaf(one.d, S[k], one.p);
        a.scan.state[static_cast<size_t>(slots[k]) * a.scan.state_stride + c] = state;
        a.scan.out[static_cast<size_t>(token) * a.scan.ld_out + c] =
            __float2bfloat16_rn(state * hx_gelu_tanh_fast(y[k] + by));
        if (a.scan.y == nullptr)
          clear_sums(a.scan.accum, a.scan.ld_accum, a.scan.channels, token, c);
      }
    }
  }
}

template <typename T>
int check_scan(const GatedScanArgs<T>& a, int dtype) {
  HX_REQUIRE(a.channels > 0 && a.ld_out >= a.channels, "hx_gated_scan: bad sizes");
  HX_REQUIRE((a.y != nullptr) != (a.accum != nullptr),
             "hx_gated_scan: give the other branch's rows or the sums of both branches");
  HX_REQUIRE(a.y == nullptr || a.ld_y >= a.channels, "hx_gated_scan: row stride too small");
  HX_REQUIRE(a.accum == nullptr || a.ld_accum >= 2 * a.channels,
             "hx_gated_scan: the sums hold both branches, the other one first");
  HX_REQUIRE(a.state != nullptr && a.y_bias != nullptr && a.out != nullptr,
             "hx_gated_scan: state, bias or output missing");
  HX_REQUIRE(dtype == HX_F32 || dtype == HX_BF16, "hx_gated_scan: unknown dtype %d", dtype);
  return HX_OK;
}

}  // namespace

// decay[t][c] = a - 1 and push[t][c] = sqrt(1 - a^2) i u with log a = -rate[c] r, r and i the
// sigmoids of block b's products with u's part b; w [blocks][2][size][size] (the rows of R,
// then of I) and u in `dtype`, everything else float32.
HX_API int hx_block_gates(const void* u, int ld_u, const void* w, const float* r_bias,
                          const float* i_bias, const float* rate, float* decay, float* push,
                          int dtype, int tokens, int blocks, int size, cudaStream_t stream) {
  HX_REQUIRE(tokens >= 0 && blocks > 0 && size > 0 && blocks <= 65535, "hx_block_gates: bad sizes");
  HX_REQUIRE(ld_u >= blocks * size, "hx_block_gates: row stride too small");
  HX_REQUIRE(r_bias && i_bias && rate && decay && push, "hx_block_gates: an operand is missing");
  if (tokens == 0) return HX_OK;
  const dim3 grid((tokens + GATE_TILE - 1) / GATE_TILE, (size + GATE_TILE - 1) / GATE_TILE, blocks);
  HX_REQUIRE(grid.y <= 65535, "hx_block_gates: blocks too large");
  if (dtype == HX_F32) {
    GateArgs<float> a{static_cast<const float*>(u), ld_u, static_cast<const float*>(w), r_bias,
                      i_bias, rate, decay, push, tokens, size, blocks * size};
    hx_launch(block_gates_kernel<float>, grid, 256, 0, stream, a);
  } else if (dtype == HX_BF16) {
    GateArgs<__nv_bfloat16> a{static_cast<const __nv_bfloat16*>(u), ld_u,
                              static_cast<const __nv_bfloat16*>(w), r_bias, i_bias, rate, decay,
                              push, tokens, size, blocks * size};
    hx_launch(block_gates_kernel<__nv_bfloat16>, grid, 256, 0, stream, a);
  } else {
    HX_REQUIRE(false, "hx_block_gates: unknown dtype %d", dtype);
  }
  HX_CHECK_LAUNCH("hx_block_gates");
  return HX_OK;
}

// out[t][c] = S gelu_tanh(y[t][c] + y_bias[c]) with S <- S + (decay S + push) over each request's
// tokens.  y [tokens][ld_y] in `dtype`, or null: the float32 sums accum [tokens][ld_accum] hold y's
// columns and, behind them, the filtered branch's; both are cleared.
HX_API int hx_gated_scan(const float* decay, const float* push, const void* y, int ld_y,
                         float* accum, int ld_accum, const float* y_bias, float* state,
                         long long state_stride, void* out, int ld_out, int dtype, int channels,
                         const int* request_start, const int* request_slot, int requests,
                         cudaStream_t stream) {
  HX_REQUIRE(requests >= 0 && requests <= 65535 && decay && push, "hx_gated_scan: bad sizes");
  if (dtype == HX_F32) {
    GatedScanArgs<float> a{decay, push, static_cast<const float*>(y), ld_y, accum, ld_accum, y_bias,
                           state, state_stride, static_cast<float*>(out), ld_out, channels,
                           request_start, request_slot};
    const int rc = check_scan(a, dtype);
    if (rc != HX_OK) return rc;
    if (requests == 0) return HX_OK;
    hx_launch(gated_scan_kernel<float>, dim3((channels + 63) / 64, requests), 64, 0, stream, a);
  } else {
    GatedScanArgs<__nv_bfloat16> a{decay, push, static_cast<const __nv_bfloat16*>(y), ld_y, accum,
                                   ld_accum, y_bias, state, state_stride,
                                   static_cast<__nv_bfloat16*>(out), ld_out, channels,
                                   request_start, request_slot};
    const int rc = check_scan(a, dtype);
    if (rc != HX_OK) return rc;
    if (requests == 0) return HX_OK;
    hx_launch(gated_scan_kernel<__nv_bfloat16>, dim3((channels + 63) / 64, requests), 64, 0, stream,
              a);
  }
  HX_CHECK_LAUNCH("hx_gated_scan");
  return HX_OK;
}

// 1 when the tiled kernels and hx_gated_recurrence_step take blocks of this size (bfloat16).
HX_API int hx_gated_recurrence_supports(int size) { return size > 0 && size % 8 == 0; }

// hx_block_gates for bfloat16 and blocks of a multiple of 8 channels, by tiles of 64 tokens of each
// request: also leaves every tile's composition in joined [tile_bound][channels] (pairs of floats)
// and every request's state before the step in before [requests][channels].  tile_bound: tokens /
// 64 + requests is always enough.
HX_API int hx_block_gates_tiled(const void* u, int ld_u, const void* w, const float* r_bias,
                                const float* i_bias, const float* rate, float* decay, float* push,
                                float* joined, const float* state, long long state_stride,
                                float* before, int blocks, int size, const int* request_start,
                                const int* request_slot, int requests, int tile_bound,
                                cudaStream_t stream) {
  HX_REQUIRE(requests >= 0 && tile_bound >= 0 && tile_bound <= 65535 && blocks > 0 &&
                 hx_gated_recurrence_supports(size),
             "hx_block_gates_tiled: %d blocks of %d channels, %d tiles are not supported", blocks, size,
             tile_bound);
  HX_REQUIRE(ld_u >= blocks * size && ld_u % 8 == 0 && (reinterpret_cast<uintptr_t>(u) & 15) == 0 &&
                 (reinterpret_cast<uintptr_t>(w) & 15) == 0 &&
                 (reinterpret_cast<uintptr_t>(joined) & 7) == 0,
             "hx_block_gates_tiled: operands must be 16-byte aligned");
  HX_REQUIRE(r_bias && i_bias && rate && decay && push && joined && state && before,
             "hx_block_gates_tiled: an operand is missing");
  if (requests == 0 || tile_bound == 0) return HX_OK;
  TiledGateArgs a{static_cast<const __nv_bfloat16*>(u), ld_u, static_cast<const __nv_bfloat16*>(w),
                  r_bias, i_bias, rate, decay, push, reinterpret_cast<float2*>(joined), state,
                  state_stride, before, request_start, request_slot, requests, size, blocks * size,
                  (size + TILE_CHANNELS - 1) / TILE_CHANNELS};
  hx_launch(tiled_gates_kernel, dim3(blocks * a.channel_tiles, tile_bound), TILE_WARPS * 32, 0, stream,
            a);
  HX_CHECK_LAUNCH("hx_block_gates_tiled");
  return HX_OK;
}

// hx_gated_scan behind hx_block_gates_tiled (bfloat16), with the same tile_bound.
HX_API int hx_gated_scan_tiled(const float* decay, const float* push, const float* joined,
                               const float* before, const void* y, int ld_y, float* accum,
                               int ld_accum, const float* y_bias, float* state,
                               long long state_stride, void* out, int ld_out, int channels,
                               const int* request_start, const int* request_slot, int requests,
                               int tile_bound, cudaStream_t stream) {
  HX_REQUIRE(requests >= 0 && tile_bound >= 0 && tile_bound <= 65535 && decay && push && joined &&
                 before && (reinterpret_cast<uintptr_t>(joined) & 7) == 0,
             "hx_gated_scan_tiled: bad sizes or an operand is missing");
  TiledScanArgs a{GatedScanArgs<__nv_bfloat16>{decay, push, static_cast<const __nv_bfloat16*>(y), ld_y,
                                               accum, ld_accum, y_bias, state, state_stride,
                                               static_cast<__nv_bfloat16*>(out), ld_out, channels,
                                               request_start, request_slot},
                  reinterpret_cast<const float2*>(joined), before, requests};
  const int rc = check_scan(a.scan, HX_BF16);
  if (rc != HX_OK) return rc;
  if (requests == 0 || tile_bound == 0) return HX_OK;
  hx_launch(tiled_scan_kernel, dim3((channels + SCAN_CHANNELS - 1) / SCAN_CHANNELS, tile_bound),
            SCAN_WARPS * 32, 0, stream, a);
  HX_CHECK_LAUNCH("hx_gated_scan_tiled");
  return HX_OK;
}

// hx_block_gates and hx_gated_scan as one kernel for a step in which every request brings exactly
// one token (bfloat16, blocks of a multiple of 8 channels).
HX_API int hx_gated_recurrence_step(const void* u, int ld_u, const void* w, const float* r_bias,
                                    const float* i_bias, const float* rate, const void* y, int ld_y,
                                    float* accum, int ld_accum, const float* y_bias, float* state,
                                    long long state_stride, void* out, int ld_out, int tokens,
                                    int blocks, int size, const int* token_request,
                                    const int* request_slot, cudaStream_t stream) {
  HX_REQUIRE(tokens >= 0 && blocks > 0 && hx_gated_recurrence_supports(size),
             "hx_gated_recurrence_step: blocks of %d channels are not supported (multiples of 8)",
             size);
  HX_REQUIRE(ld_u >= blocks * size && ld_u % 8 == 0 && (reinterpret_cast<uintptr_t>(u) & 15) == 0 &&
                 (reinterpret_cast<uintptr_t>(w) & 15) == 0,
             "hx_gated_recurrence_step: operands must be 16-byte aligned");
  HX_REQUIRE(r_bias && i_bias && rate, "hx_gated_recurrence_step: an operand is missing");
  StepArgs a{static_cast<const __nv_bfloat16*>(u), ld_u, static_cast<const __nv_bfloat16*>(w),
             r_bias, i_bias, rate,
             GatedScanArgs<__nv_bfloat16>{nullptr, nullptr, static_cast<const __nv_bfloat16*>(y),
                                          ld_y, accum, ld_accum, y_bias, state, state_stride,
                                          static_cast<__nv_bfloat16*>(out), ld_out, blocks * size,
                                          nullptr, request_slot},
             token_request, tokens, size, (size + STEP_CHANNELS - 1) / STEP_CHANNELS};
  const int rc = check_scan(a.scan, HX_BF16);
  if (rc != HX_OK) return rc;
  if (tokens == 0) return HX_OK;
  const int grid = blocks * a.tiles;
  if (tokens <= 8) {
    hx_launch(gated_recurrence_step_kernel<1>, grid, STEP_WARPS * 32, 0, stream, a);
  } else if (tokens <= 16) {
    hx_launch(gated_recurrence_step_kernel<2>, grid, STEP_WARPS * 32, 0, stream, a);
  } else if (tokens <= 32) {
    hx_launch(gated_recurrence_step_kernel<4>, grid, STEP_WARPS * 32, 0, stream, a);
  } else {
    hx_launch(gated_recurrence_step_kernel<8>, grid, STEP_WARPS * 32, 0, stream, a);
  }
  HX_CHECK_LAUNCH("hx_gated_recurrence_step");
  return HX_OK;
}
