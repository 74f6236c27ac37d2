// A matrix state with one decay per head and token, walked 64 tokens at a time on the tensor cores
// (bfloat16 rows):
//
//     S_t = e^(d_t) S_(t-1) + p_t k_t v_t',     o_t = S_t' (c q_t),       d_t <= 0
//
// with v_t followed by a 1, so that S has one more column, the decayed sum of p_t k_t alone.  With L_t the
// sum of d over the chunk up to t, a chunk that starts from S_0 gives
//
//     o_t  = c e^(L_t) S_0' q_t  +  sum_(s <= t) P_ts v_s,      P_ts = c (q_t . k_s) e^(L_t - L_s) p_s
//     S_64 = e^(L_64) S_0 + sum_s w_s k_s v_s',                 w_s = e^(L_64 - L_s) p_s
//
// Every exponent is a difference of decays between two tokens of the chunk, never positive.
//
//   * chunk_weights_kernel, all chunks at once: P (stored as two bfloat16 terms, about 16 bits of each
//     value) and, in place of d and p, the factors c e^(L_t) and w_s.
//   * chunk_states_kernel, one CTA per (request, head, block of columns), chunk after chunk: a warp keeps
//     S' for 16 columns and up to 128 coordinates of the key in registers, as the accumulators of
//     mma.sync (64 where the grid leaves room).  The layout of two neighbouring accumulator tiles is that of an A operand, so S' goes
//     into o' = S' Q' without leaving the registers (as two bfloat16 terms; it stays float32 itself), and
//     the update S' += (w V)' K adds into the same registers (w v as two terms).  Keys of more than 128
//     coordinates are shared out to several warps whose parts of o are summed through shared memory.
//     The next chunk's rows are on their way while one is worked on.
//
// The state lies in the request's row as the other recurrences keep theirs (hx_scan.cuh).
#include "hx_mma.cuh"
#include "hx_scan.cuh"

namespace {

constexpr int CHUNK = 64;
constexpr int ROW_PAD = 8;              // elements behind a staged row: rows start on different banks
constexpr int WEIGHT_COLUMNS = 2 * CHUNK;    // of a token's row of P: 64 hi terms, 64 lo terms

struct ChunkArgs {
  const __nv_bfloat16* q;    // [tokens, ld], already offset; heads * dim columns
  const __nv_bfloat16* k;
  const __nv_bfloat16* v;    // heads * vdim columns
  int ld;
  float* decay;              // [heads, ld_gates]: d, then c e^L
  float* push;               // [heads, ld_gates]: p, then w
  float* total;              // [heads, ld_gates]: e^(L_64) at a chunk's first token
  int ld_gates;
  __nv_bfloat16* weights;    // [heads, ld_gates, WEIGHT_COLUMNS]
  float q_scale;
  float* state;
  long long state_stride;
  int head_stride;
  float* o;                  // [tokens, heads * vdim]
  float* extra;              // [heads, ld_gates]: the last column's output
  const int* request_start;
  const int* request_slot;
  int requests, heads, dim, vdim, parts;
  int padded;                // dim in whole steps of the warps' shares
  int key_warps, column_warps, stages;
};

__device__ __forceinline__ void copy_4(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}

// A thread's way through 64 rows of `pieces` 16-byte pieces: it keeps its place in the row and goes down
// `row_step` rows at a time; threads that do not fit a whole row of the block's pass stand by.
struct PieceWalk {
  int row, piece, row_step;
  __device__ __forceinline__ explicit PieceWalk(int pieces_of_row) {
    const int pieces = max(pieces_of_row, 1);
    row_step = static_cast<int>(blockDim.x) / pieces;
    row = static_cast<int>(threadIdx.x) / pieces;
    piece = static_cast<int>(threadIdx.x) - row * pieces;
    if (row >= row_step) row = CHUNK;
  }
};

// 64 rows into shared memory with `stride` elements a row; rows from `live` on are zeros.
__device__ __forceinline__ void copy_rows(const PieceWalk& walk, __nv_bfloat16* dst, int stride,
                                          const __nv_bfloat16* src, size_t ld, int live) {
  uint32_t to = hx_shared_address(dst) + 2 * (walk.row * stride + 8 * walk.piece);
  const uint32_t to_step = 2 * walk.row_step * stride;
  const __nv_bfloat16* from = src + walk.row * ld + 8 * walk.piece;
  const size_t from_step = walk.row_step * ld;
  if (live == CHUNK) {
#pragma unroll 4
    for (int row = walk.row; row < CHUNK; row += walk.row_step) {
      hx_cp_async_16(to, from, 16);
      to += to_step;
      from += from_step;
    }
  } else {
    for (int row = walk.row; row < CHUNK; row += walk.row_step) {
      const bool there = row < live;
      hx_cp_async_16(to, there ? from : src, there ? 16 : 0);
      to += to_step;
      from += from_step;
    }
  }
}

// zeros behind the copied columns, once: the copies never touch them
__device__ __forceinline__ void clear_columns(__nv_bfloat16* dst, int stride, int from, int to) {
  const int width = to - from;
  for (int i = threadIdx.x; i < CHUNK * width; i += blockDim.x) {
    const int row = i / width;
    dst[row * stride + from + i - row * width] = __float2bfloat16_rn(0.0f);
  }
}

// grid (chunks of the step, heads), 128 threads: a warp takes 16 of the chunk's tokens
__global__ __launch_bounds__(128) void chunk_weights_kernel(const ChunkArgs a) {
  extern __shared__ uint4 shared_pieces[];
  __shared__ float level[CHUNK], add[CHUNK];
  hx_pdl_prologue();
  int chunk, chunks;
  const int request = hx_find_query_tile(a.request_start, a.requests, 1, CHUNK, blockIdx.x, chunk, chunks);
  if (request < 0) return;
  const int head = blockIdx.y;
  const int first = a.request_start[request] + chunk * CHUNK;
  const int live = min(CHUNK, a.request_start[request + 1] - first);
  const int stride = a.padded + ROW_PAD;
  __nv_bfloat16* queries = reinterpret_cast<__nv_bfloat16*>(shared_pieces);
  __nv_bfloat16* keys = queries + CHUNK * stride;
  const size_t ld = a.ld;
  const PieceWalk walk(a.dim >> 3);
  copy_rows(walk, queries, stride, a.q + first * ld + head * a.dim, ld, live);
  copy_rows(walk, keys, stride, a.k + first * ld + head * a.dim, ld, live);
  hx_cp_async_commit();
  if (a.padded > a.dim) {
    clear_columns(queries, stride, a.dim, a.padded);
    clear_columns(keys, stride, a.dim, a.padded);
  }
  const size_t gates = static_cast<size_t>(head) * a.ld_gates + first;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if (warp == 0) {
    // sums of the decays' logarithms, two neighbouring tokens a lane
    const float d0 = 2 * lane < live ? a.decay[gates + 2 * lane] : 0.0f;
    const float d1 = 2 * lane + 1 < live ? a.decay[gates + 2 * lane + 1] : 0.0f;
    float sum = d0 + d1;
#pragma unroll
    for (int offset = 1; offset < 32; offset <<= 1) {
      const float other = __shfl_up_sync(0xffffffffu, sum, offset);
      if (lane >= offset) sum += other;
    }
    const float first_level = sum - d1;
    level[2 * lane] = first_level;
    level[2 * lane + 1] = sum;
    const float all = __shfl_sync(0xffffffffu, sum, 31);
    const float p0 = 2 * lane < live ? a.push[gates + 2 * lane] : 0.0f;
    const float p1 = 2 * lane + 1 < live ? a.push[gates + 2 * lane + 1] : 0.0f;
    add[2 * lane] = p0;
    add[2 * lane + 1] = p1;
    if (2 * lane < live) {
      a.decay[gates + 2 * lane] = a.q_scale * expf(first_level);
      a.push[gates + 2 * lane] = expf(all - first_level) * p0;
    }
    if (2 * lane + 1 < live) {
      a.decay[gates + 2 * lane + 1] = a.q_scale * expf(sum);
      a.push[gates + 2 * lane + 1] = expf(all - sum) * p1;
    }
    if (lane == 0) a.total[gates] = expf(all);
  }
  hx_cp_async_wait<0>();
  __syncthreads();
  // sums of tokens 16 warp .. + 15 against the tiles of 8 tokens that do not lie behind them
  float acc[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[n][j] = 0.0f;
  const int tiles = 2 * warp + 2;
  const int matrix = lane >> 3, in_matrix = lane & 7;
  const uint32_t a_at = hx_shared_address(queries + (16 * warp + (matrix & 1) * 8 + in_matrix) * stride + (matrix >> 1) * 8);
  const uint32_t b_at = hx_shared_address(keys + ((matrix >> 1) * 8 + in_matrix) * stride + (matrix & 1) * 8);
  for (int step = 0; step < a.padded / 16; ++step) {
    uint32_t af[4];
    hx_ldmatrix_x4(af, a_at + 32 * step);
#pragma unroll
    for (int n = 0; n < 8; n += 2) {
      if (n < tiles) {
        uint32_t bf[4];
        hx_ldmatrix_x4(bf, b_at + 2 * (8 * n * stride + 16 * step));
        hx_mma_bf16(acc[n], af, bf[0], bf[1]);
        hx_mma_bf16(acc[n + 1], af, bf[2], bf[3]);
      }
    }
  }
  const int row = lane >> 2, column = 2 * (lane & 3);
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t = 16 * warp + row + 8 * half;
    if (t >= live) continue;
    __nv_bfloat16* out = a.weights + (gates + t) * WEIGHT_COLUMNS;
    const float at = level[t];
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const int s = 8 * n + column;
      float w0 = 0.0f, w1 = 0.0f;
      if (s <= t) w0 = acc[n][2 * half] * a.q_scale * (expf(at - level[s]) * add[s]);
      if (s + 1 <= t) w1 = acc[n][2 * half + 1] * a.q_scale * (expf(at - level[s + 1]) * add[s + 1]);
      uint32_t hi, lo;
      hx_split_bf16(w0, w1, hi, lo);
      *reinterpret_cast<uint32_t*>(out + s) = hi;
      *reinterpret_cast<uint32_t*>(out + CHUNK + s) = lo;
    }
  }
}

constexpr int WEIGHT_STRIDE = WEIGHT_COLUMNS + ROW_PAD;
constexpr int PART_STRIDE = 20;       // floats a token's 16 columns take: no bank is hit twice
constexpr int PART_FLOATS = CHUNK * PART_STRIDE;

// Shared memory of chunk_states_kernel, in bytes: `stages` times [queries | keys | weights | values |
// factors, pushes, total], the warps' parts of o, the weighted values (when they are shared).
struct StatesLayout {
  int rows_bytes, stage_bytes, parts_bytes, weighted_bytes, bytes;
  __host__ __device__ StatesLayout(int padded, int key_warps, int column_warps, int stages) {
    rows_bytes = 2 * CHUNK * (2 * (padded + ROW_PAD) + WEIGHT_STRIDE + 16 * column_warps + ROW_PAD);
    stage_bytes = rows_bytes + 4 * (2 * CHUNK + 4);
    parts_bytes = 4 * key_warps * column_warps * PART_FLOATS;
    // (one warp weights the values for itself, two do it twice: cheaper than handing them over)
    weighted_bytes = key_warps > 2 ? 2 * CHUNK * (32 * column_warps + ROW_PAD) : 0;
    bytes = stages * stage_bytes + parts_bytes + weighted_bytes;
  }
};

// STEPS: steps of 16 key coordinates that a warp keeps; SHARED_VALUES: the weighted values are made once
// for all warps of a column
template <int STEPS, bool SHARED_VALUES>
__global__ __launch_bounds__(256) void chunk_states_kernel(const ChunkArgs a) {
  extern __shared__ uint4 shared_pieces[];
  hx_pdl_prologue();
  const int request = blockIdx.x, head = blockIdx.y;
  const int start = a.request_start[request];
  const int count = a.request_start[request + 1] - start;
  if (count <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int key_warp = warp % a.key_warps, column_warp = warp / a.key_warps;
  const int row = lane >> 2, pair = 2 * (lane & 3);
  const int matrix = lane >> 3, in_matrix = lane & 7;
  const int columns = a.vdim + 1, block_columns = 16 * a.column_warps;
  const int column0 = blockIdx.z * block_columns;
  const int copied = max(0, min(a.vdim - column0, block_columns));     // columns that are values
  const int stride = a.padded + ROW_PAD, value_stride = block_columns + ROW_PAD;
  const int weighted_stride = 2 * block_columns + ROW_PAD;
  const StatesLayout layout(a.padded, a.key_warps, a.column_warps, a.stages);
  char* base = reinterpret_cast<char*>(shared_pieces);
  float* parts = reinterpret_cast<float*>(base + a.stages * layout.stage_bytes);
  __nv_bfloat16* weighted = reinterpret_cast<__nv_bfloat16*>(base + a.stages * layout.stage_bytes + layout.parts_bytes);
  auto queries_of = [&](int stage) { return reinterpret_cast<__nv_bfloat16*>(base + stage * layout.stage_bytes); };
  const size_t ld = a.ld;
  const PieceWalk key_walk(a.dim >> 3), weight_walk(WEIGHT_COLUMNS >> 3), value_walk(copied >> 3);
  auto fetch = [&](int chunk, int stage) {
    const int first = start + chunk * CHUNK;
    const int live = min(CHUNK, count - chunk * CHUNK);
    const size_t gates = static_cast<size_t>(head) * a.ld_gates + first;
    __nv_bfloat16* queries = queries_of(stage);
    __nv_bfloat16* keys = queries + CHUNK * stride;
    __nv_bfloat16* weights = keys + CHUNK * stride;
    __nv_bfloat16* values = weights + CHUNK * WEIGHT_STRIDE;
    copy_rows(key_walk, queries, stride, a.q + first * ld + head * a.dim, ld, live);
    copy_rows(key_walk, keys, stride, a.k + first * ld + head * a.dim, ld, live);
    copy_rows(weight_walk, weights, WEIGHT_STRIDE, a.weights + gates * WEIGHT_COLUMNS, WEIGHT_COLUMNS, live);
    if (copied > 0)
      copy_rows(value_walk, values, value_stride, a.v + first * ld + head * a.vdim + column0, ld, live);
    float* floats = reinterpret_cast<float*>(base + stage * layout.stage_bytes + layout.rows_bytes);
    for (int i = threadIdx.x; i < 2 * CHUNK + 1; i += blockDim.x) {
      const int t = i & (CHUNK - 1);
      const bool there = i == 2 * CHUNK || t < live;
      const float* source = (i < CHUNK ? a.decay : i < 2 * CHUNK ? a.push : a.total) + gates;
      copy_4(hx_shared_address(floats + i), there ? source + t : source, there ? 4 : 0);
    }
    hx_cp_async_commit();
  };
  // what the copies leave alone: zeros behind the keys' coordinates; behind the values a one (the
  // last column of S) and zeros
  for (int stage = 0; stage < a.stages; ++stage) {
    __nv_bfloat16* queries = queries_of(stage);
    __nv_bfloat16* values = queries + CHUNK * (2 * stride + WEIGHT_STRIDE);
    if (a.padded > a.dim) {
      clear_columns(queries, stride, a.dim, a.padded);
      clear_columns(queries + CHUNK * stride, stride, a.dim, a.padded);
    }
    for (int i = threadIdx.x; i < CHUNK * (block_columns - copied); i += blockDim.x) {
      const int t = i / (block_columns - copied), c = copied + i - t * (block_columns - copied);
      values[t * value_stride + c] = __float2bfloat16_rn(column0 + c == a.vdim ? 1.0f : 0.0f);
    }
  }
  fetch(0, 0);

  // the warp's part of S': columns column0 + 16 column_warp + row (+ 8), key coordinates
  // 16 STEPS key_warp + 8 n + pair (+ 1)
  float* s_state = a.state + static_cast<size_t>(a.request_slot[request]) * a.state_stride +
                   static_cast<size_t>(head) * a.head_stride;
  const int lanes = columns * a.parts;
  const int my_column = column0 + 16 * column_warp + row, my_dim = 16 * STEPS * key_warp + pair;
  float S[2 * STEPS][4];
#pragma unroll
  for (int n = 0; n < 2 * STEPS; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = my_column + 8 * (j >> 1), d = my_dim + 8 * n + (j & 1);
      S[n][j] = c < columns && d < a.dim
                    ? s_state[static_cast<size_t>(d & 15) * lanes + c * a.parts + (d >> 4)] : 0.0f;
    }
  // which of the chunk's steps of 16 tokens are this warp's among those that share its columns
  bool own_step[CHUNK / 16];
#pragma unroll
  for (int step = 0; step < CHUNK / 16; ++step) own_step[step] = step % a.key_warps == key_warp;
  // offsets of the lane's rows in the operands
  const uint32_t q_lane = 2 * (((matrix >> 1) * 8 + in_matrix) * stride + (matrix & 1) * 8 + 16 * STEPS * key_warp);
  const uint32_t k_lane = 2 * (((matrix & 1) * 8 + in_matrix) * stride + (matrix >> 1) * 8 + 16 * STEPS * key_warp);
  const uint32_t w_lane = 2 * (((matrix >> 1) * 8 + in_matrix) * WEIGHT_STRIDE + (matrix & 1) * 8);
  const uint32_t v_lane = 2 * (((matrix >> 1) * 8 + in_matrix) * value_stride + 16 * column_warp + (matrix & 1) * 8);
  const uint32_t weighted_at = hx_shared_address(weighted) +
      2 * (((matrix >> 1) * 8 + in_matrix) * weighted_stride + 16 * column_warp + (matrix & 1) * 8);
  float* my_part = parts + warp * PART_FLOATS + pair * PART_STRIDE + row;     // [column_warp][key_warp]
  const int chunks = (count + CHUNK - 1) / CHUNK;
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const int stage = a.stages == 2 ? chunk & 1 : 0;
    hx_cp_async_wait<0>();
    __syncthreads();
    if (a.stages == 2 && chunk + 1 < chunks) fetch(chunk + 1, stage ^ 1);
    const uint32_t queries = hx_shared_address(queries_of(stage));
    const uint32_t keys = queries + 2 * CHUNK * stride;
    const uint32_t weights = keys + 2 * CHUNK * stride;
    const uint32_t values = weights + 2 * CHUNK * WEIGHT_STRIDE;
    const float* factor = reinterpret_cast<const float*>(base + stage * layout.stage_bytes + layout.rows_bytes);
    const float* push = factor + CHUNK;
    const float total = factor[2 * CHUNK];

    if constexpr (SHARED_VALUES) {
      // w v as two terms, a piece of 8 columns of a token per thread and round
      const __nv_bfloat16* raw = queries_of(stage) + CHUNK * (2 * stride + WEIGHT_STRIDE);
      const int pieces = 2 * a.column_warps;
      for (int i = threadIdx.x; i < CHUNK * pieces; i += blockDim.x) {
        const int t = i / pieces, c = 8 * (i - t * pieces);
        const uint4 packed = *reinterpret_cast<const uint4*>(raw + t * value_stride + c);
        const float w = push[t];
        uint4 hi, lo;
        const __nv_bfloat162* x = reinterpret_cast<const __nv_bfloat162*>(&packed);
        uint32_t* h = reinterpret_cast<uint32_t*>(&hi);
        uint32_t* l = reinterpret_cast<uint32_t*>(&lo);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float2 v = __bfloat1622float2(x[k]);
          hx_split_bf16(v.x * w, v.y * w, h[k], l[k]);
        }
        *reinterpret_cast<uint4*>(weighted + t * weighted_stride + c) = hi;
        *reinterpret_cast<uint4*>(weighted + t * weighted_stride + block_columns + c) = lo;
      }
    }
    // o' [16 columns x 64 tokens]: the state in front of the chunk, products into eight accumulators
    // before any of them is needed again
    float out[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int j = 0; j < 4; ++j) out[n][j] = 0.0f;
#pragma unroll
    for (int step = 0; step < STEPS; ++step) {
      uint32_t b[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n) hx_ldmatrix_x4(b[n], queries + q_lane + 2 * (16 * n * stride + 16 * step));
      uint32_t s_hi[4], s_lo[4];
      hx_split_bf16(S[2 * step][0], S[2 * step][1], s_hi[0], s_lo[0]);
      hx_split_bf16(S[2 * step][2], S[2 * step][3], s_hi[1], s_lo[1]);
      hx_split_bf16(S[2 * step + 1][0], S[2 * step + 1][1], s_hi[2], s_lo[2]);
      hx_split_bf16(S[2 * step + 1][2], S[2 * step + 1][3], s_hi[3], s_lo[3]);
#pragma unroll
      for (int n = 0; n < 8; ++n) hx_mma_bf16(out[n], s_hi, b[n >> 1][2 * (n & 1)], b[n >> 1][2 * (n & 1) + 1]);
#pragma unroll
      for (int n = 0; n < 8; ++n) hx_mma_bf16(out[n], s_lo, b[n >> 1][2 * (n & 1)], b[n >> 1][2 * (n & 1) + 1]);
    }
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const float2 f = *reinterpret_cast<const float2*>(factor + 8 * n + pair);
      out[n][0] *= f.x; out[n][1] *= f.y;
      out[n][2] *= f.x; out[n][3] *= f.y;
    }
    // the chunk's own tokens
#pragma unroll
    for (int step = 0; step < CHUNK / 16; ++step) {
      if (!own_step[step]) continue;
      uint32_t v[4];
      hx_ldmatrix_x4_trans(v, values + v_lane + 2 * (16 * step * value_stride));
#pragma unroll
      for (int term = 0; term < 2; ++term)
#pragma unroll
        for (int n = 2 * step; n < 8; n += 2) {
          uint32_t b[4];
          hx_ldmatrix_x4(b, weights + w_lane + 2 * (8 * n * WEIGHT_STRIDE + CHUNK * term + 16 * step));
          hx_mma_bf16(out[n], v, b[0], b[1]);
          hx_mma_bf16(out[n + 1], v, b[2], b[3]);
        }
    }
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int j = 0; j < 4; ++j) my_part[(8 * n + (j & 1)) * PART_STRIDE + 8 * (j >> 1)] = out[n][j];
    __syncthreads();
    {
      // the parts of the warps that share the columns, summed in their order; four columns of a token
      // per thread and round
      const int first = start + chunk * CHUNK, live = min(CHUNK, count - chunk * CHUNK);
      const int quads = 4 * a.column_warps;
      for (int i = threadIdx.x; i < live * quads; i += blockDim.x) {
        const int t = i / quads, c = 4 * (i - t * quads);
        if (column0 + c >= columns) continue;
        const float* from = parts + (c >> 4) * a.key_warps * PART_FLOATS + t * PART_STRIDE + (c & 15);
        float4 sum = *reinterpret_cast<const float4*>(from);
        for (int other = 1; other < a.key_warps; ++other) {
          const float4 x = *reinterpret_cast<const float4*>(from + other * PART_FLOATS);
          sum.x += x.x; sum.y += x.y; sum.z += x.z; sum.w += x.w;
        }
        if (column0 + c < a.vdim) {
          *reinterpret_cast<float4*>(a.o + static_cast<size_t>(first + t) * (a.heads * a.vdim) +
                                     head * a.vdim + column0 + c) = sum;
        } else {
          a.extra[static_cast<size_t>(head) * a.ld_gates + first + t] = sum.x;
        }
      }
    }
    // the state behind the chunk
#pragma unroll
    for (int n = 0; n < 2 * STEPS; ++n)
#pragma unroll
      for (int j = 0; j < 4; ++j) S[n][j] *= total;
#pragma unroll
    for (int step = 0; step < CHUNK / 16; ++step) {
      uint32_t v_hi[4], v_lo[4];
      if constexpr (SHARED_VALUES) {
        hx_ldmatrix_x4_trans(v_hi, weighted_at + 2 * (16 * step * weighted_stride));
        hx_ldmatrix_x4_trans(v_lo, weighted_at + 2 * (16 * step * weighted_stride + block_columns));
      } else {
        uint32_t v[4];
        hx_ldmatrix_x4_trans(v, values + v_lane + 2 * (16 * step * value_stride));
        const float2 w0 = *reinterpret_cast<const float2*>(push + 16 * step + pair);
        const float2 w1 = *reinterpret_cast<const float2*>(push + 16 * step + 8 + pair);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v[i]));
          const float2 w = i < 2 ? w0 : w1;
          hx_split_bf16(x.x * w.x, x.y * w.y, v_hi[i], v_lo[i]);
        }
      }
      constexpr int GROUP = STEPS < 4 ? STEPS : 4;      // pairs of tiles in flight
#pragma unroll
      for (int group = 0; group < STEPS; group += GROUP) {
        uint32_t b[GROUP][4];
#pragma unroll
        for (int n = 0; n < GROUP; ++n)
          if (group + n < STEPS)
            hx_ldmatrix_x4_trans(b[n], keys + k_lane + 2 * (16 * step * stride + 16 * (group + n)));
#pragma unroll
        for (int n = 0; n < 2 * GROUP; ++n)
          if (group + (n >> 1) < STEPS)
            hx_mma_bf16(S[2 * group + n], v_hi, b[n >> 1][2 * (n & 1)], b[n >> 1][2 * (n & 1) + 1]);
#pragma unroll
        for (int n = 0; n < 2 * GROUP; ++n)
          if (group + (n >> 1) < STEPS)
            hx_mma_bf16(S[2 * group + n], v_lo, b[n >> 1][2 * (n & 1)], b[n >> 1][2 * (n & 1) + 1]);
      }
    }
    if (a.stages == 1) {
      __syncthreads();
      if (chunk + 1 < chunks) fetch(chunk + 1, 0);
    }
  }
#pragma unroll
  for (int n = 0; n < 2 * STEPS; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = my_column + 8 * (j >> 1), d = my_dim + 8 * n + (j & 1);
      if (c < columns && d < a.dim)
        s_state[static_cast<size_t>(d & 15) * lanes + c * a.parts + (d >> 4)] = S[n][j];
    }
}

constexpr int MAX_SHARED = 227 * 1024;

int weights_shared(int padded) { return 2 * 2 * CHUNK * (padded + ROW_PAD); }
template <int STEPS, bool SHARED_VALUES>
int launch_states(const ChunkArgs& a, dim3 grid, int threads, int shared, cudaStream_t stream) {
  if (cudaFuncSetAttribute(chunk_states_kernel<STEPS, SHARED_VALUES>,
                           cudaFuncAttributeMaxDynamicSharedMemorySize, MAX_SHARED) != cudaSuccess) {
    hx_set_error("hx_state_chunks: the device refuses %d bytes of shared memory", MAX_SHARED);
    return HX_ERR_LAUNCH;
  }
  hx_launch(chunk_states_kernel<STEPS, SHARED_VALUES>, grid, threads, shared, stream, a);
  return HX_OK;
}

}  // namespace

// 1: heads of these sizes run here (bfloat16); else they take the token-by-token scan.
HX_API int hx_state_chunks_supports(int dim, int vdim) {
  return dim > 0 && vdim > 0 && dim % 8 == 0 && vdim % 8 == 0 && dim <= 512 && parts_for(dim) > 0 ? 1 : 0;
}

// Elements (bfloat16) of the scratch `weights` for rows of ld_gates tokens.
HX_API long long hx_state_chunks_scratch(int heads, int ld_gates) {
  return static_cast<long long>(heads) * ld_gates * WEIGHT_COLUMNS;
}

// See the head of this file.  q, k, v bfloat16 columns of rows [tokens, ld] (16-byte aligned, heads * dim
// and heads * vdim columns); decay and push [heads, ld_gates] float32 hold d and p and are overwritten;
// total [heads, ld_gates] and weights (hx_state_chunks_scratch) are scratch; state rows as
// hx_matrix_lstm_state_floats lays them out (head_stride floats a head); o float32 [tokens, heads * vdim],
// extra [heads, ld_gates].  tiles: chunks of 64 tokens in the step, request by request.
HX_API int hx_state_chunks(const void* q, const void* k, const void* v, int ld, float* decay, float* push,
                           float* total, int ld_gates, void* weights, float q_scale, float* state,
                           long long state_stride, int head_stride, float* o, float* extra,
                           const int* request_start, const int* request_slot, int requests, int tiles,
                           int heads, int dim, int vdim, cudaStream_t stream) {
  HX_REQUIRE(hx_state_chunks_supports(dim, vdim), "hx_state_chunks: heads of %d by %d are not supported",
             dim, vdim);
  HX_REQUIRE(requests >= 0 && tiles >= requests && heads > 0 && heads <= 65535 && ld % 8 == 0 && ld_gates > 0,
             "hx_state_chunks: bad sizes");
  HX_REQUIRE(((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) |
               reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(weights)) & 15) == 0,
             "hx_state_chunks: rows are not 16-byte aligned");
  HX_REQUIRE(head_stride >= state_floats(vdim + 1, dim) &&
                 state_stride >= static_cast<long long>(heads) * head_stride,
             "hx_state_chunks: state rows too short");
  if (requests == 0) return HX_OK;
  // how a head's matrix is dealt: as few columns a CTA and as few key coordinates a warp as leave the
  // grid within one wave of the GPU (a request's chunks follow one another, so the time is a CTA's)
  const int steps_in_all = (dim + 15) / 16;
  auto blocks_for = [&](int warps) { return (vdim + 1 + 16 * warps - 1) / (16 * warps); };
  int most_steps = steps_in_all <= 16 ? 4 : 8, column_warps = 2;
  if (static_cast<long long>(requests) * heads * blocks_for(2) > hx_device_sm_count()) {
    if (steps_in_all > 8) most_steps = 8;
    if (steps_in_all <= 16) column_warps = 4;
  }
  const int key_warps = (steps_in_all + most_steps - 1) / most_steps;
  int steps = (steps_in_all + key_warps - 1) / key_warps;
  if (steps > 2) steps = (steps + 1) / 2 * 2;         // 1, 2, 4, 6, 8
  const int padded = 16 * steps * key_warps;
  int stages = 2;
  if (StatesLayout(padded, key_warps, column_warps, stages).bytes > MAX_SHARED) stages = 1;
  const int shared = StatesLayout(padded, key_warps, column_warps, stages).bytes;
  HX_REQUIRE(shared <= MAX_SHARED && weights_shared(padded) <= MAX_SHARED,
             "hx_state_chunks: heads of %d do not fit shared memory", dim);
  const ChunkArgs a{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(k),
                    static_cast<const __nv_bfloat16*>(v), ld, decay, push, total, ld_gates,
                    static_cast<__nv_bfloat16*>(weights), q_scale, state, state_stride, head_stride, o,
                    extra, request_start, request_slot, requests, heads, dim, vdim, parts_for(dim), padded,
                    key_warps, column_warps, stages};
  if (cudaFuncSetAttribute(chunk_weights_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                           MAX_SHARED - 1024) != cudaSuccess) {
    hx_set_error("hx_state_chunks: the device refuses %d bytes of shared memory", MAX_SHARED - 1024);
    return HX_ERR_LAUNCH;
  }
  hx_launch(chunk_weights_kernel, dim3(tiles, heads), 128, weights_shared(padded), stream, a);
  const dim3 grid(requests, heads, blocks_for(column_warps));
  const int threads = 32 * key_warps * column_warps;
  const bool shares = key_warps > 2;      // (then a warp keeps three steps at least)
  int rc;
  switch (steps) {
    case 1: rc = launch_states<1, false>(a, grid, threads, shared, stream); break;
    case 2: rc = launch_states<2, false>(a, grid, threads, shared, stream); break;
    case 4: rc = shares ? launch_states<4, true>(a, grid, threads, shared, stream)
                        : launch_states<4, false>(a, grid, threads, shared, stream); break;
    case 6: rc = shares ? launch_states<6, true>(a, grid, threads, shared, stream)
                        : launch_states<6, false>(a, grid, threads, shared, stream); break;
    default: rc = shares ? launch_states<8, true>(a, grid, threads, shared, stream)
                         : launch_states<8, false>(a, grid, threads, shared, stream); break;
  }
  if (rc != HX_OK) return rc;
  hx_count_launches(1);
  HX_CHECK_LAUNCH("hx_state_chunks");
  return HX_OK;
}
