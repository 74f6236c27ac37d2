// The matrix memory of an mLSTM layer: per head a matrix S [dim x vdim] and a vector n [dim],
//
//     m_t = max(f_t + m_(t-1), i_t)
//     S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t',   n_t likewise with k_t alone
//     o_t = S_t' q_t / (max(|n_t . q_t|, exp(-m_t)) + floor)
//
// with i = cap tanh(zi / cap) the logarithm of the input gate, f = log sigmoid(cap tanh(zf / cap)) that
// of the forget gate, and m, the running maximum, zero at admission.  Behind it each head's o over
// its root mean square, times a weight, times sigmoid(g).
//
// n is one more column of S whose value is always 1: a head keeps [dim x (vdim + 1)], dealt to lanes
// and laid out in the state row like the other recurrences' matrices (hx_scan.cuh); behind the heads'
// matrices the row holds m per head.
//
//   * gates (prompt portions): one CTA per (request, head) turns the gates' float32 sums into, per
//     token, the decay's logarithm d = f + (m_(t-1) - m_t), the input weight exp(i - m) and exp(-m).
//     The maximum is an associative composition of (sum of f, best i so far), scanned 256 tokens at
//     a time.  d is taken from the rounded maxima that S is scaled by: the difference of two
//     neighbouring maxima is exact, so a rounding of m (which may be larger than f itself when a
//     gate hardly forgets) is a change of scale that d undoes, not an error of S.
//   * scan: token by token, any sizes, both engines; a decode step takes its gates here.  Prompt
//     portions in bfloat16 go through hx_state_chunks instead.
//   * finish: division, norm, weight and gate; in a decode step also the new maximum, and the
//     projection's sums are cleared.
#include "hx_scan.cuh"

namespace {

__device__ __forceinline__ float log_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_forget_gate(float z, float cap) {
  const float x = cap * tanhf(z / cap);
  return fminf(x, 0.0f) - log1pf(expf(-fabsf(x)));
}

// ------------------------------------------------------------------------------ gates

constexpr int GATE_THREADS = 256;

struct LstmGateArgs {
  const float* sums;        // [tokens, ld]: input gates of the heads, then forget gates
  int ld;
  const float* bias;        // [2 * heads]
  float cap;
  float* log_decay;         // [heads, ld_out], and so are the other two
  float* push;
  float* level;             // exp(-m)
  int ld_out;
  float* maxima;            // per slot: [heads]
  long long state_stride;
  const int* request_start;
  const int* request_slot;
  int heads;
};

// (sum of log forgets, best log input so far), first one, then the other
__device__ __forceinline__ void compose(float& sum, float& best, float sum_before, float best_before) {
  best = fmaxf(best_before + sum, best);
  sum += sum_before;
}

// grid (requests, heads)
__global__ __launch_bounds__(GATE_THREADS) void lstm_gates_kernel(const LstmGateArgs a) {
  constexpr int WARPS = GATE_THREADS / 32;
  __shared__ float warp_sum[WARPS], warp_best[WARPS], warp_last[WARPS];
  hx_pdl_prologue();
  const int request = blockIdx.x, head = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int start = a.request_start[request];
  const int count = a.request_start[request + 1] - start;
  float* kept = a.maxima + static_cast<size_t>(a.request_slot[request]) * a.state_stride + head;
  float before = *kept;                    // the maximum in front of the stretch
  const float in_bias = a.bias[head], forget_bias = a.bias[a.heads + head];
  for (int base = 0; base < count; base += GATE_THREADS) {
    const int t = base + threadIdx.x;
    const bool live = t < count;
    float log_in = -INFINITY, log_forget = 0.0f;       // an element that changes nothing
    if (live) {
      const float* z = a.sums + static_cast<size_t>(start + t) * a.ld;
      log_in = log_input_gate(z[head] + in_bias, a.cap);
      log_forget = log_forget_gate(z[a.heads + head] + forget_bias, a.cap);
    }
    float sum = log_forget, best = log_in;
#pragma unroll
    for (int offset = 1; offset < 32; offset <<= 1) {
      const float other_sum = __shfl_up_sync(0xffffffffu, sum, offset);
      const float other_best = __shfl_up_sync(0xffffffffu, best, offset);
      if (lane >= offset) compose(sum, best, other_sum, other_best);
    }
    if (lane == 31) { warp_sum[warp] = sum; warp_best[warp] = best; }
    __syncthreads();
    // the maximum in front of this warp's tokens
    float m = before;
    for (int w = 0; w < warp; ++w) m = fmaxf(m + warp_sum[w], warp_best[w]);
    const float m_front = m;
    m = fmaxf(m_front + sum, best);
    // dead lanes (behind the portion) repeat the last maximum: their element changes nothing
    if (lane == 31) warp_last[warp] = m;
    float m_before = __shfl_up_sync(0xffffffffu, m, 1);
    __syncthreads();
    if (lane == 0) m_before = warp == 0 ? before : warp_last[warp - 1];
    if (live) {
      const size_t at = static_cast<size_t>(head) * a.ld_out + start + t;
      a.log_decay[at] = fminf(log_forget + (m_before - m), 0.0f);
      a.push[at] = expf(log_in - m);
      a.level[at] = expf(-m);
    }
    before = warp_last[WARPS - 1];
    __syncthreads();
  }
  if (threadIdx.x == 0) *kept = before;
}

// ------------------------------------------------------------------------------- scan

template <typename T>
struct LstmArgs {
  const T* rows;            // [tokens, ld]: q | k | v | g
  int ld;
  const float* accum;       // the same as float32 sums, with the gates' columns behind; or null
  int ld_accum;
  float q_scale, floor, cap, eps;
  const float* bias;        // [2 * heads] of the gates (decode steps)
  const float* log_decay;   // [heads, ld_gates], see LstmGateArgs (prompt portions)
  const float* push;
  const float* level;
  int ld_gates;
  const float* gate_sums;   // [tokens, ld_gate_sums]: decode steps, the gates' columns
  int ld_gate_sums;
  float* state;             // per slot: heads x head_stride | maxima [heads]
  long long state_stride;
  int head_stride;
  float* o;                 // [tokens, heads * vdim]
  float* weight;            // [heads, ld_gates]: n . q
  const float* norm;        // [heads * vdim]
  T* out;                   // [tokens, ld_out]
  int ld_out;
  float* clear;             // the accumulator to clear, or null
  int clear_width;
  const int* request_start;
  const int* request_slot;
  const int* token_request;
  int tokens, heads, dim, vdim;
  int parts, block_lanes, tile, per_token;
};

// element c of a token's row, sums rounded as the projection's own store would have
template <typename T>
__device__ __forceinline__ float lstm_row(const LstmArgs<T>& a, size_t token, int c) {
  if (a.accum != nullptr) return hx_to_float<T>(hx_from_float<T>(a.accum[token * a.ld_accum + c]));
  return hx_to_float<T>(a.rows[token * a.ld + c]);
}

// a decode step's maximum, from the state and the token's gate sums
template <typename T>
__device__ __forceinline__ void one_gate(const LstmArgs<T>& a, size_t token, int head, float before,
                                         float& m, float& log_decay, float& push) {
  const float* z = a.gate_sums + token * a.ld_gate_sums;
  const float log_in = log_input_gate(z[head] + a.bias[head], a.cap);
  const float log_forget = log_forget_gate(z[a.heads + head] + a.bias[a.heads + head], a.cap);
  m = fmaxf(log_forget + before, log_in);
  log_decay = fminf(log_forget + (before - m), 0.0f);
  push = expf(log_in - m);
}

// grid (requests, heads, blocks of columns); see hx_scan.cuh for the dealing
template <typename T, bool ONE_TOKEN>
__global__ __launch_bounds__(SCAN_THREADS, ONE_TOKEN ? 3 : HX_SCAN_CTAS)
void matrix_lstm_scan_kernel(const LstmArgs<T> a) {
  constexpr int RPT = 16;
  constexpr int STRIDE = run_stride<RPT>();
  constexpr bool EXACT = sizeof(T) == 4;      // the float32 engine, see decayed_add_exact
  extern __shared__ float4 shared4[];
  float* shared = reinterpret_cast<float*>(shared4);
  hx_pdl_prologue();
  const int request = blockIdx.x, head = blockIdx.y;
  const int start = a.request_start[request];
  const int count = ONE_TOKEN ? 1 : a.request_start[request + 1] - start;
  const int parts = a.parts, dim = a.dim, vdim = a.vdim;
  const int columns = vdim + 1;               // the last one is n
  const int lane = blockIdx.z * a.block_lanes + threadIdx.x;
  const int column = lane / parts;
  const int part = lane - column * parts;
  const bool live = column < columns && threadIdx.x < a.block_lanes;
  // staged per token: q, k (parts runs each), the block's values, decay, push
  const int run = parts * STRIDE;
  const int per_token = a.per_token;
  const int lanes = columns * parts;
  const int first_column = blockIdx.z * a.block_lanes / parts;
  const int block_columns = min(a.block_lanes / parts, columns - first_column);
  float* row_state = a.state + static_cast<size_t>(a.request_slot[request]) * a.state_stride;
  float* s_state = row_state + static_cast<size_t>(head) * a.head_stride;
  float S[RPT];
  float carry[EXACT ? RPT : 1];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    S[i] = (live && part * RPT + i < dim) ? s_state[static_cast<size_t>(i) * lanes + lane] : 0.0f;
    carry[EXACT ? i : 0] = 0.0f;
  }
  for (int i = threadIdx.x; i < (ONE_TOKEN ? 1 : a.tile) * per_token; i += blockDim.x) shared[i] = 0.0f;
  const int q_at = head * dim, k_at = (a.heads + head) * dim;
  const int v_at = 2 * a.heads * dim + head * vdim;
  for (int base = 0; base < count; base += a.tile) {
    const int here = min(a.tile, count - base);
    const size_t first = static_cast<size_t>(start + base);
    __syncthreads();
    stage<ONE_TOKEN>(shared, per_token, here, dim,
          [&](int t, int e) { return lstm_row(a, first + t, q_at + e) * a.q_scale; }, padded<RPT>);
    stage<ONE_TOKEN>(shared + run, per_token, here, dim,
          [&](int t, int e) { return lstm_row(a, first + t, k_at + e); }, padded<RPT>);
    stage<ONE_TOKEN>(shared + 2 * run, per_token, here, block_columns,
          [&](int t, int e) {
            const int c = first_column + e;
            return c < vdim ? lstm_row(a, first + t, v_at + c) : 1.0f;
          },
          [](int e) { return e; });
    float* gates = shared + per_token - 2;
    for (int t = threadIdx.x; t < here; t += blockDim.x) {
      float log_decay, push;
      if (ONE_TOKEN) {
        float m;
        one_gate(a, first, head, row_state[static_cast<size_t>(a.heads) * a.head_stride + head], m,
                 log_decay, push);
      } else {
        const size_t at = static_cast<size_t>(head) * a.ld_gates + first + t;
        log_decay = a.log_decay[at];
        push = a.push[at];
      }
      gates[t * per_token] = EXACT ? expm1f(log_decay) : expf(log_decay);
      gates[t * per_token + 1] = push;
    }
    __syncthreads();
#pragma unroll 1
    for (int t = 0; t < here; ++t) {
      const float* row = shared + t * per_token;
      const float4* q4 = reinterpret_cast<const float4*>(row + part * STRIDE);
      const float4* k4 = reinterpret_cast<const float4*>(row + run + part * STRIDE);
      const float decay = row[per_token - 2];         // EXACT: the decay minus one
      const float u = live ? row[2 * run + column - first_column] * row[per_token - 1] : 0.0f;
      float sum0 = 0.0f, sum1 = 0.0f;
#pragma unroll
      for (int c = 0; c < RPT / 4; ++c) {
        const float4 qv = q4[c];
        const float4 kv = k4[c];
        if constexpr (EXACT) {
          decayed_add_exact(S[4 * c + 0], carry[4 * c + 0], decay, kv.x * u);
          decayed_add_exact(S[4 * c + 1], carry[4 * c + 1], decay, kv.y * u);
          decayed_add_exact(S[4 * c + 2], carry[4 * c + 2], decay, kv.z * u);
          decayed_add_exact(S[4 * c + 3], carry[4 * c + 3], decay, kv.w * u);
          sum0 = fmaf(S[4 * c + 0] + carry[4 * c + 0], qv.x, sum0);
          sum1 = fmaf(S[4 * c + 1] + carry[4 * c + 1], qv.y, sum1);
          sum0 = fmaf(S[4 * c + 2] + carry[4 * c + 2], qv.z, sum0);
          sum1 = fmaf(S[4 * c + 3] + carry[4 * c + 3], qv.w, sum1);
        } else {
          S[4 * c + 0] = fmaf(decay, S[4 * c + 0], kv.x * u);
          S[4 * c + 1] = fmaf(decay, S[4 * c + 1], kv.y * u);
          S[4 * c + 2] = fmaf(decay, S[4 * c + 2], kv.z * u);
          S[4 * c + 3] = fmaf(decay, S[4 * c + 3], kv.w * u);
          sum0 = fmaf(S[4 * c + 0], qv.x, sum0);
          sum1 = fmaf(S[4 * c + 1], qv.y, sum1);
          sum0 = fmaf(S[4 * c + 2], qv.z, sum0);
          sum1 = fmaf(S[4 * c + 3], qv.w, sum1);
        }
      }
      float sum = sum0 + sum1;
      for (int offset = parts >> 1; offset > 0; offset >>= 1)
        sum += __shfl_xor_sync(0xffffffffu, sum, offset);
      if (live && part == 0) {
        if (column < vdim) {
          a.o[(first + t) * (static_cast<size_t>(a.heads) * vdim) + head * vdim + column] = sum;
        } else {
          a.weight[static_cast<size_t>(head) * a.ld_gates + first + t] = sum;
        }
      }
    }
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < RPT; ++i)
      if (part * RPT + i < dim)
        s_state[static_cast<size_t>(i) * lanes + lane] = EXACT ? S[i] + carry[EXACT ? i : 0] : S[i];
  }
}

// ----------------------------------------------------------------------------- finish

// A warp takes a head of a token; grid (tokens, ceil(heads / FINISH_WARPS)).
constexpr int FINISH_WARPS = 4;

template <typename T, bool ONE_TOKEN>
__global__ __launch_bounds__(FINISH_WARPS * 32) void matrix_lstm_finish_kernel(const LstmArgs<T> a) {
  hx_pdl_prologue();
  const size_t token = blockIdx.x;
  const int head = blockIdx.y * FINISH_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (head >= a.heads) return;
  const int vdim = a.vdim;
  const size_t at = static_cast<size_t>(head) * a.ld_gates + token;
  float level;
  if (ONE_TOKEN) {
    float* maxima = a.state + static_cast<size_t>(a.request_slot[a.token_request[token]]) * a.state_stride +
                    static_cast<size_t>(a.heads) * a.head_stride;
    float m, log_decay, push;
    one_gate(a, token, head, maxima[head], m, log_decay, push);
    level = expf(-m);
    __syncwarp();
    if (lane == 0) maxima[head] = m;
  } else {
    level = a.level[at];
  }
  const float inverse = 1.0f / (fmaxf(fabsf(a.weight[at]), level) + a.floor);
  const float* o = a.o + token * (static_cast<size_t>(a.heads) * vdim) + head * vdim;
  float sum = 0.0f;
  constexpr int HELD = 16;
  float held[HELD];
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int c = lane + 32 * i;
    held[i] = c < vdim ? o[c] * inverse : 0.0f;
    sum = fmaf(held[i], held[i], sum);
  }
  for (int c = lane + 32 * HELD; c < vdim; c += 32) {
    const float v = o[c] * inverse;
    sum = fmaf(v, v, sum);
  }
#pragma unroll
  for (int offset = 16; offset > 0; offset >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, offset);
  const float unit = 1.0f / sqrtf(sum / static_cast<float>(vdim) + a.eps);
  const int g_at = a.heads * (2 * a.dim + vdim) + head * vdim;
  T* out = a.out + token * a.ld_out + head * vdim;
  auto put = [&](int c, float v) {
    out[c] = hx_from_float<T>(v * unit * a.norm[head * vdim + c] * hx_sigmoid(lstm_row(a, token, g_at + c)));
    if (a.clear != nullptr) a.clear[token * a.ld_accum + g_at + c] = 0.0f;
  };
#pragma unroll
  for (int i = 0; i < HELD; ++i)
    if (lane + 32 * i < vdim) put(lane + 32 * i, held[i]);
  for (int c = lane + 32 * HELD; c < vdim; c += 32) put(c, o[c] * inverse);
  if (a.clear != nullptr) {
    // the head's share of q, k, v (read by the scan, which is done) and its two gates
    float* row = a.clear + token * a.ld_accum;
    for (int c = lane; c < a.dim; c += 32) {
      row[head * a.dim + c] = 0.0f;
      row[(a.heads + head) * a.dim + c] = 0.0f;
    }
    for (int c = lane; c < vdim; c += 32) row[2 * a.heads * a.dim + head * vdim + c] = 0.0f;
    if (lane == 0) {
      const int gates = 2 * a.heads * (a.dim + vdim);
      row[gates + head] = 0.0f;
      row[gates + a.heads + head] = 0.0f;
    }
  }
}

// The same in pieces of four numbers: GROUP threads take a head of a token.
__device__ __forceinline__ float4 row_quad(const LstmArgs<float>& a, size_t token, int c) {
  return *reinterpret_cast<const float4*>((a.accum != nullptr ? a.accum + token * a.ld_accum
                                                              : a.rows + token * a.ld) + c);
}
__device__ __forceinline__ float4 row_quad(const LstmArgs<__nv_bfloat16>& a, size_t token, int c) {
  uint2 packed;
  if (a.accum != nullptr) {
    const float4 v = *reinterpret_cast<const float4*>(a.accum + token * a.ld_accum + c);
    *reinterpret_cast<__nv_bfloat162*>(&packed.x) = __floats2bfloat162_rn(v.x, v.y);
    *reinterpret_cast<__nv_bfloat162*>(&packed.y) = __floats2bfloat162_rn(v.z, v.w);
  } else {
    packed = *reinterpret_cast<const uint2*>(a.rows + token * a.ld + c);
  }
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&packed.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&packed.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void put_quad(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put_quad(__nv_bfloat16* p, float4 v) {
  uint2 packed;
  *reinterpret_cast<__nv_bfloat162*>(&packed.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&packed.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = packed;
}
// the gate's sigmoid: results stored in bfloat16 take the hardware exponential
template <typename T> __device__ __forceinline__ float gate_of(float x) {
  return sizeof(T) == 4 ? hx_sigmoid(x) : __fdividef(1.0f, 1.0f + __expf(-x));
}

template <typename T, bool ONE_TOKEN, int GROUP>
__global__ __launch_bounds__(128) void matrix_lstm_finish_quads_kernel(const LstmArgs<T> a) {
  __shared__ float scratch[32];
  hx_pdl_prologue();
  const size_t token = blockIdx.x;
  const int head = blockIdx.y * (128 / GROUP) + threadIdx.x / GROUP, lane = threadIdx.x & (GROUP - 1);
  if (GROUP == 32 && head >= a.heads) return;          // a block of one group has its head
  const int vdim = a.vdim, quads = vdim >> 2;
  const float4* o = reinterpret_cast<const float4*>(a.o + token * (static_cast<size_t>(a.heads) * vdim) + head * vdim);
  const int g_at = a.heads * (2 * a.dim + vdim) + head * vdim;
  float4 held[2], gate[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int q = lane + GROUP * i;
    held[i] = q < quads ? o[q] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    gate[i] = q < quads ? row_quad(a, token, g_at + 4 * q) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  const size_t at = static_cast<size_t>(head) * a.ld_gates + token;
  float level, m = 0.0f;
  float* kept = nullptr;
  if (ONE_TOKEN) {
    kept = a.state + static_cast<size_t>(a.request_slot[a.token_request[token]]) * a.state_stride +
           static_cast<size_t>(a.heads) * a.head_stride + head;
    float log_decay, push;
    one_gate(a, token, head, *kept, m, log_decay, push);
    level = expf(-m);
  } else {
    level = a.level[at];
  }
  const float inverse = 1.0f / (fmaxf(fabsf(a.weight[at]), level) + a.floor);
  float sum = 0.0f;
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    held[i].x *= inverse; held[i].y *= inverse; held[i].z *= inverse; held[i].w *= inverse;
    sum = fmaf(held[i].x, held[i].x, sum); sum = fmaf(held[i].y, held[i].y, sum);
    sum = fmaf(held[i].z, held[i].z, sum); sum = fmaf(held[i].w, held[i].w, sum);
  }
  if (GROUP == 32) {
#pragma unroll
    for (int offset = 16; offset > 0; offset >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, offset);
  } else {
    sum = hx_block_sum(sum, scratch);
  }
  const float unit = 1.0f / sqrtf(sum / static_cast<float>(vdim) + a.eps);
  T* out = a.out + token * a.ld_out + head * vdim;
  const float4* norm = reinterpret_cast<const float4*>(a.norm + head * vdim);
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int q = lane + GROUP * i;
    if (q >= quads) continue;
    const float4 w = norm[q];
    put_quad(out + 4 * q, make_float4(held[i].x * unit * w.x * gate_of<T>(gate[i].x),
                                      held[i].y * unit * w.y * gate_of<T>(gate[i].y),
                                      held[i].z * unit * w.z * gate_of<T>(gate[i].z),
                                      held[i].w * unit * w.w * gate_of<T>(gate[i].w)));
  }
  // everybody has read the old maximum and the gates' sums (the sum above synchronised the group)
  if (ONE_TOKEN && lane == 0) *kept = m;
  if (a.clear != nullptr) {
    float* row = a.clear + token * a.ld_accum;
    const float4 zeros = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    for (int q = lane; q < a.dim >> 2; q += GROUP) {
      put_quad(row + head * a.dim + 4 * q, zeros);
      put_quad(row + (a.heads + head) * a.dim + 4 * q, zeros);
    }
    for (int q = lane; q < quads; q += GROUP) {
      put_quad(row + 2 * a.heads * a.dim + head * vdim + 4 * q, zeros);
      put_quad(row + g_at + 4 * q, zeros);
    }
    if (lane == 0) {
      const int gates = 2 * a.heads * (a.dim + vdim);
      row[gates + head] = 0.0f;
      row[gates + a.heads + head] = 0.0f;
    }
  }
}

template <typename T, bool ONE_TOKEN>
void launch_finish(const LstmArgs<T>& a, cudaStream_t stream) {
  auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  if (a.vdim % 4 == 0 && a.dim % 4 == 0 && a.vdim <= 1024 && a.ld_out % 4 == 0 && aligned(a.o) &&
      aligned(a.norm) && aligned(a.out) && aligned(a.rows) && aligned(a.accum) &&
      (a.accum != nullptr ? a.ld_accum : a.ld) % 4 == 0) {
    if (a.vdim <= 256) {
      hx_launch(matrix_lstm_finish_quads_kernel<T, ONE_TOKEN, 32>, dim3(a.tokens, (a.heads + 3) / 4), 128, 0,
                stream, a);
    } else {
      hx_launch(matrix_lstm_finish_quads_kernel<T, ONE_TOKEN, 128>, dim3(a.tokens, a.heads), 128, 0, stream, a);
    }
    return;
  }
  hx_launch(matrix_lstm_finish_kernel<T, ONE_TOKEN>,
            dim3(a.tokens, (a.heads + FINISH_WARPS - 1) / FINISH_WARPS), FINISH_WARPS * 32, 0, stream, a);
}

template <typename T>
int run_matrix_lstm(LstmArgs<T> a, int requests, bool scan, cudaStream_t stream) {
  const int columns = a.vdim + 1;
  a.parts = parts_for(a.dim);
  a.block_lanes = min(columns, SCAN_THREADS / a.parts) * a.parts;
  a.per_token = staged_floats(2, a.dim, a.block_lanes / a.parts + 2);
  a.tile = tile_for(a.per_token);
  HX_REQUIRE(a.tile >= 1, "hx_matrix_lstm: a token's vectors do not fit shared memory");
  if (scan) {
    const int threads = (a.block_lanes + 31) / 32 * 32;
    const int column_blocks = (columns * a.parts + a.block_lanes - 1) / a.block_lanes;
    const dim3 grid(requests, a.heads, column_blocks);
    const size_t one_bytes = static_cast<size_t>(a.per_token) * sizeof(float);
    if (a.gate_sums != nullptr) {
      hx_launch(matrix_lstm_scan_kernel<T, true>, grid, threads, one_bytes, stream, a);
    } else {
      hx_launch(matrix_lstm_scan_kernel<T, false>, grid, threads, a.tile * one_bytes, stream, a);
    }
    hx_count_launches(1);
  }
  if (a.gate_sums != nullptr) {
    launch_finish<T, true>(a, stream);
  } else {
    launch_finish<T, false>(a, stream);
  }
  return HX_OK;
}

}  // namespace

// Floats of a request's state row: `heads` matrices [dim x (vdim + 1)] and the maxima; 0: the sizes
// have no kernel.
HX_API int hx_matrix_lstm_state_floats(int heads, int dim, int vdim) {
  if (heads <= 0 || dim <= 0 || vdim <= 0 || parts_for(dim) == 0) return 0;
  return heads * (state_floats(vdim + 1, dim) + 1);
}

// Gates of a step's prompt portions: sums float32 [tokens, ld] (input gates of the heads, then
// forget gates), bias [2 * heads]; log_decay, push and level [heads, ld_out] float32, token index
// last.  `state`: the state rows (the maxima behind the heads' matrices are read and updated).
HX_API int hx_matrix_lstm_gates(const float* sums, int ld, const float* bias, float cap,
                                float* log_decay, float* push, float* level, int ld_out, float* state,
                                long long state_stride, const int* request_start,
                                const int* request_slot, int requests, int tokens, int heads, int dim,
                                int vdim, cudaStream_t stream) {
  HX_REQUIRE(requests >= 0 && tokens >= 0 && heads > 0 && heads <= 65535 && ld >= 2 * heads &&
                 ld_out >= tokens && cap > 0.0f && hx_matrix_lstm_state_floats(heads, dim, vdim) > 0,
             "hx_matrix_lstm_gates: bad sizes");
  HX_REQUIRE(state_stride >= hx_matrix_lstm_state_floats(heads, dim, vdim),
             "hx_matrix_lstm_gates: state rows too short");
  if (requests == 0 || tokens == 0) return HX_OK;
  float* maxima = state + static_cast<size_t>(heads) * state_floats(vdim + 1, dim);
  const LstmGateArgs a{sums, ld, bias, cap, log_decay, push, level, ld_out, maxima, state_stride,
                       request_start, request_slot, heads};
  hx_launch(lstm_gates_kernel, dim3(requests, heads), GATE_THREADS, 0, stream, a);
  HX_CHECK_LAUNCH("hx_matrix_lstm_gates");
  return HX_OK;
}

// The recurrence and what follows it.  rows [tokens, ld] in `dtype`, or accum float32 sums [tokens,
// ld_accum] (rounded into `dtype` when read, and cleared): q [heads * dim] | k | v [heads * vdim] | g,
// accum with the 2 * heads gate columns behind.  gate_sums not null: a decode step (one token per
// request), gates from these columns; null: gates from hx_matrix_lstm_gates' arrays [heads,
// ld_gates].  scan 0: o float32 [tokens, heads * vdim] and weight [heads, ld_gates] hold the recurrence's
// results already (hx_state_chunks); else they are scratch.  out [tokens, ld_out] in `dtype`.
HX_API int hx_matrix_lstm(const void* rows, int ld, float* accum, int ld_accum, int dtype,
                          const float* gate_sums, int ld_gate_sums, const float* bias, float cap,
                          const float* log_decay, const float* push, const float* level, int ld_gates,
                          int scan, float q_scale, float floor, const float* norm, float eps, float* state,
                          long long state_stride, float* o, float* weight, void* out, int ld_out,
                          const int* token_request, const int* request_start, const int* request_slot,
                          int requests, int tokens, int heads, int dim, int vdim, cudaStream_t stream) {
  HX_REQUIRE(requests >= 0 && tokens >= requests && heads > 0 && heads <= 65535 && dim > 0 && vdim > 0 &&
                 cap > 0.0f && eps > 0.0f && floor >= 0.0f && ld_out >= heads * vdim && ld_gates >= tokens,
             "hx_matrix_lstm: bad sizes");
  HX_REQUIRE(parts_for(dim) > 0, "hx_matrix_lstm: heads of %d are more than %d", dim, 32 * 16);
  const int columns = 2 * heads * (dim + vdim);
  HX_REQUIRE(scan || gate_sums == nullptr, "hx_matrix_lstm: a decode step scans");
  HX_REQUIRE((rows != nullptr) != (accum != nullptr),
             "hx_matrix_lstm: give the projected rows or their sums");
  HX_REQUIRE(rows == nullptr || ld >= columns, "hx_matrix_lstm: row stride too small");
  HX_REQUIRE(accum == nullptr || ld_accum >= columns + 2 * heads,
             "hx_matrix_lstm: accumulator stride too small");
  HX_REQUIRE(gate_sums != nullptr ? tokens == requests && ld_gate_sums >= 2 * heads
                                  : log_decay != nullptr && push != nullptr && level != nullptr,
             "hx_matrix_lstm: gates missing");
  HX_REQUIRE(state_stride >= hx_matrix_lstm_state_floats(heads, dim, vdim),
             "hx_matrix_lstm: state rows too short");
  if (requests == 0) return HX_OK;
  const int head_stride = state_floats(vdim + 1, dim);
  int rc;
  if (dtype == HX_F32) {
    rc = run_matrix_lstm(LstmArgs<float>{static_cast<const float*>(rows), ld, accum, ld_accum, q_scale,
                                         floor, cap, eps, bias, log_decay, push, level, ld_gates,
                                         gate_sums, ld_gate_sums, state, state_stride, head_stride, o,
                                         weight, norm, static_cast<float*>(out), ld_out, accum,
                                         columns + 2 * heads, request_start, request_slot,
                                         token_request, tokens, heads, dim, vdim, 0, 0, 0, 0},
                         requests, scan != 0, stream);
  } else if (dtype == HX_BF16) {
    rc = run_matrix_lstm(LstmArgs<__nv_bfloat16>{
                             static_cast<const __nv_bfloat16*>(rows), ld, accum, ld_accum, q_scale, floor,
                             cap, eps, bias, log_decay, push, level, ld_gates, gate_sums, ld_gate_sums,
                             state, state_stride, head_stride, o, weight, norm,
                             static_cast<__nv_bfloat16*>(out), ld_out, accum, columns + 2 * heads,
                             request_start, request_slot, token_request, tokens, heads, dim, vdim, 0, 0,
                             0, 0},
                         requests, scan != 0, stream);
  } else {
    HX_REQUIRE(false, "hx_matrix_lstm: unknown dtype %d", dtype);
  }
  if (rc != HX_OK) return rc;
  HX_CHECK_LAUNCH("hx_matrix_lstm");
  return HX_OK;
}
