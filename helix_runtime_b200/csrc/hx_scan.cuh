// What the recurrences with a matrix state share: how a head's matrix is dealt to lanes and laid
// out in a request's state row, how the tokens' vectors are staged in shared memory, and the
// float32 engine's step that carries its own rounding.
//
// A thread owns a column of S (one value coordinate) and a run of consecutive rows of it; `parts`
// neighbouring lanes share a column and add their partial sums with shuffles.  In memory the
// matrix is [row % run][column][row / run].
#pragma once

#include "hx_common.cuh"

namespace {

__device__ __forceinline__ float softplus(float x) {
  return x > 20.0f ? x : log1pf(expf(x));
}

// One step S <- decay * S + add of a recurrence in the float32 engine.  A decay close to one
// cannot be told from its neighbours in float32 (their spacing is 6e-8), and a head that hardly
// forgets multiplies a thousand such decays over a long prompt: the roundings add up like a
// random walk and show in the logits of late positions.  So the decay arrives as d = decay - 1
// (taken with expm1f, which keeps its digits), the step is S + (d S + add), and the rounding of
// that sum (a two-sum recovers it) is carried beside S in `carry`, which decays like S.  What
// reads the state reads S + carry; the state row holds S + carry rounded once.
__device__ __forceinline__ void decayed_add_exact(float& S, float& carry, float d, float add) {
  const float t = fmaf(d, S, add);
  const float sum = S + t;
  const float shadow = sum - S;
  const float error = (S - (sum - shadow)) + (t - shadow);
  carry = fmaf(d, carry, carry) + error;
  S = sum;
}

// Rows of a column that one lane keeps.  A pure function of the row count, because the state's
// order in memory follows from it.  Sixteen for every size: runs of 4 and 8 (more lanes and
// CTAs per head, each staging the tokens' vectors again) were measured at the sizes of a 7B
// model's layers and lost, 2.0 against 1.26 ms for 2,048 tokens of a state-space layer and
// 190 against 68 us for a decode step of 64 requests of a time-mixing layer.
__host__ __device__ constexpr int rows_per_thread(int rows) { return rows > 0 ? 16 : 16; }
// Threads of a CTA at most.  A head whose columns need more is cut into blocks of columns
// (blockIdx.z), each a CTA of its own with the same tokens staged.
constexpr int SCAN_THREADS = 256;
// CTAs the compiler makes room for on an SM (it bounds the registers of a thread).
#ifndef HX_SCAN_CTAS
#define HX_SCAN_CTAS 2
#endif
#ifndef HX_SCAN_TILE_KB
#define HX_SCAN_TILE_KB 24
#endif

// Rows of a staged vector are kept in runs of RPT (one lane's share); runs of eight and more
// have four floats of padding behind them, so that the lanes of a warp, which read different
// runs with 16-byte loads, fall on different banks.
template <int RPT> constexpr int run_stride() { return RPT + (RPT >= 8 ? 4 : 0); }
template <int RPT>
__device__ __forceinline__ int padded(int n) { return n + (n / RPT) * (RPT >= 8 ? 4 : 0); }

// One vector of `length` elements for each of `tokens` tokens: dst[t * stride + place(e)] =
// load(t, e).  Warps take tokens, lanes take elements (consecutive addresses), four loads in
// flight per lane; nothing divides.
template <bool ONE_TOKEN, typename Load, typename Place>
__device__ __forceinline__ void stage(float* dst, int stride, int tokens, int length, Load load,
                                      Place place) {
  if (ONE_TOKEN) {      // a decode step: one vector, one load per thread and round
    for (int e = threadIdx.x; e < length; e += blockDim.x) dst[place(e)] = load(0, e);
    return;
  }
  const int warp = threadIdx.x >> 5;
  const int warps = blockDim.x >> 5;
  const int lane = threadIdx.x & 31;
  for (int t = warp; t < tokens; t += warps) {
    float* row = dst + t * stride;
    for (int first = lane; first < length; first += 128) {
      float v[4];
#pragma unroll
      for (int u = 0; u < 4; ++u)
        if (first + 32 * u < length) v[u] = load(t, first + 32 * u);
#pragma unroll
      for (int u = 0; u < 4; ++u)
        if (first + 32 * u < length) row[place(first + 32 * u)] = v[u];
    }
  }
}

// lanes that share a column: the smallest power of two that leaves a lane at most
// rows_per_thread(rows) rows; 0 when even a whole warp would not do
int parts_for(int rows) {
  for (int parts = 1; parts <= 32; parts <<= 1)
    if (parts * rows_per_thread(rows) >= rows) return parts;
  return 0;
}

int state_floats(int columns, int rows) {
  const int parts = parts_for(rows);
  return parts * rows_per_thread(rows) * columns;
}

// floats staged per token: `vectors` vectors of `rows` rows in padded runs, and `plain` more;
// a multiple of four, so that every token's runs start on 16 bytes
int staged_floats(int vectors, int rows, int plain) {
  const int rpt = rows_per_thread(rows);
  return (vectors * parts_for(rows) * (rpt + (rpt >= 8 ? 4 : 0)) + plain + 3) / 4 * 4;
}

// tokens staged per tile: a tile of at most HX_SCAN_TILE_KB kilobytes (below the 48 KB a CTA gets
// without asking), so that several CTAs share an SM
int tile_for(int floats_per_token) {
  const int budget = HX_SCAN_TILE_KB * 1024 / 4;
  int tile = budget / floats_per_token;
  if (tile > 32) tile = 32;
  return tile;
}

}  // namespace
