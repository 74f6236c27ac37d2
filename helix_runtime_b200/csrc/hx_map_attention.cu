// What an attention layer with several score maps per head does between its projection and the
// cache, and behind the attention.
//
// hx_filtered_heads.  A row of the projection is [q: heads * maps * dim | k: kv_heads * maps * dim | v:
// kv_heads * vdim | further columns].  Every channel gets its bias and passes a causal filter over
// time (`taps` weights, the last on the token itself, zeros in front of the sequence); every map of
// every query and key head then passes an RMS norm over its `dim` coordinates (one weight for all)
// and is rotated by its position over its first `rot` coordinates, neighbouring pairs, with
// cosines and sines from a table; values are filtered only.
//
// All maps of a key head share ONE cached row [k_1 | k_2 | ...] beside the head's value row, and the
// query row of map m is zero outside that map's place in it.  So the maps of a head are ordinary
// query heads of a grouped attention whose key/value heads are the model's own: the scores of map m
// are q_m . k_m, no attention kernel knows of maps, and a key and its value are cached once.
// Queries leave in rows of row_dim per (head, map), keys and values go to their pages.
//
// A unit is a map of a query or key head, or a value head.  Heads in whole 16-byte pieces: a lane owns
// one piece (8 channels) of a run of consecutive tokens, 2^n neighbouring lanes a unit; other even
// sizes: a warp owns a unit, a lane pairs of channels; any sizes: the same without a run.  Either way
// the norm is a sum over lanes and a rotation stays inside a lane.  Only the first taps - 1 tokens of a request's portion reach behind it, into
// the request's state (its last taps - 1 inputs): whoever has the portion's first token works on all
// of them and then writes the new state, so one owner per (request, unit) touches it.
//
// hx_map_difference.  With a1, a2 the attention results of a head's two maps: o = a1 - lambda a2,
// over sqrt(mean(o^2) + eps), times `scale`, times sigmoid(g); a warp per (token, head).
#include "hx_common.cuh"

namespace {

template <typename T>
struct FilteredHeadsArgs {
  const T* raw;             // [tokens, ld_raw], or
  int ld_raw;
  const float* accum;       // float32 sums [tokens, ld_accum], rounded as the projection's store would
  int ld_accum;
  const float* bias;        // [channels] or null
  const float* filter;      // [channels, taps]
  float* state;             // per slot: [taps - 1, channels]
  long long state_stride;
  int taps, channels;
  const float* q_norm;      // [dim] or null: no norm
  const float* k_norm;
  float eps;
  const float* cosine;      // [table_rows, rot / 2]
  const float* sine;
  int rot, table_rows;
  T* out;                   // [tokens, ld_out]: heads * maps rows of row_dim
  int ld_out;
  T* k_cache;
  T* v_cache;
  const int* positions;
  const int* token_request;
  const int* request_slot;
  const int* request_start;
  const int* block_tables;
  int table_stride;
  int tokens, run;
  int heads, kv_heads, maps, dim, vdim, row_dim;   // kv_heads 0: queries only
  int page_size, num_pages;
  int* status;
};

// which unit a warp owns
struct Unit {
  int kind;       // 0 query map, 1 key map, 2 value
  int head, map;  // head: query head (0), key/value head (1, 2)
  int column;     // its first channel
  int width;
};

template <typename T>
__device__ __forceinline__ Unit unit_of(const FilteredHeadsArgs<T>& a, int index) {
  Unit u;
  const int q_units = a.heads * a.maps, k_units = a.kv_heads * a.maps;
  if (index < q_units) {
    u.kind = 0; u.head = index / a.maps; u.map = index - u.head * a.maps;
    u.column = index * a.dim; u.width = a.dim;
  } else if (index < q_units + k_units) {
    const int k = index - q_units;
    u.kind = 1; u.head = k / a.maps; u.map = k - u.head * a.maps;
    u.column = index * a.dim; u.width = a.dim;
  } else {
    u.kind = 2; u.head = index - q_units - k_units; u.map = 0;
    u.column = (q_units + k_units) * a.dim + u.head * a.vdim; u.width = a.vdim;
  }
  return u;
}

template <typename T>
__device__ __forceinline__ float warp_sum(T v) {
#pragma unroll
  for (int offset = 16; offset > 0; offset >>= 1) v += __shfl_xor_sync(0xffffffffu, v, offset);
  return v;
}

// The unit's filtered channels of one token (`y[2 i], y[2 i + 1]` the lane's pair lane + 32 i): norm,
// rotation, store.  WIDE: even widths and aligned rows, a pair is one access.
template <typename T, int PAIRS, bool WIDE>
__device__ __forceinline__ void finish_unit(const FilteredHeadsArgs<T>& a, const Unit& u, int token,
                                            int position, int table_row, float (&y)[2 * PAIRS]) {
  const int lane = threadIdx.x & 31;
  if (u.kind != 2) {
    const float* weight = u.kind == 0 ? a.q_norm : a.k_norm;
    if (weight != nullptr) {
      float sum = 0.0f;
#pragma unroll
      for (int i = 0; i < 2 * PAIRS; ++i) sum = fmaf(y[i], y[i], sum);
      const float unit = 1.0f / sqrtf(warp_sum(sum) / static_cast<float>(u.width) + a.eps);
#pragma unroll
      for (int i = 0; i < PAIRS; ++i) {
        const int c = 2 * (lane + 32 * i);
        if (c < u.width) y[2 * i] *= unit * weight[c];
        if (c + 1 < u.width) y[2 * i + 1] *= unit * weight[c + 1];
      }
    }
    if (a.rot > 0) {
      if (position >= a.table_rows) {
        if (lane == 0 && a.status != nullptr) atomicOr(a.status, HX_FLAG_BAD_POSITION);
        return;
      }
      const int half = a.rot >> 1;
      const float* cosine = a.cosine + static_cast<size_t>(position) * half;
      const float* sine = a.sine + static_cast<size_t>(position) * half;
#pragma unroll
      for (int i = 0; i < PAIRS; ++i) {
        const int p = lane + 32 * i;
        if (p < half) {
          const float c = cosine[p], s = sine[p], first = y[2 * i], second = y[2 * i + 1];
          y[2 * i] = first * c - second * s;
          y[2 * i + 1] = second * c + first * s;
        }
      }
    }
  }
  // where it goes: `place(d)` is the address of coordinate d of the row the unit lies in
  const int R = a.row_dim;
  const int own = u.kind == 2 ? 0 : u.map * a.dim;          // the unit's first coordinate in it
  if (u.kind == 0) {
    T* row = a.out + static_cast<size_t>(token) * a.ld_out + (u.head * a.maps + u.map) * R;
    if constexpr (WIDE) {
      auto pair = [&](int c, float first, float second) {
        if constexpr (sizeof(T) == 2) {
          *reinterpret_cast<__nv_bfloat162*>(row + c) = __floats2bfloat162_rn(first, second);
        } else {
          *reinterpret_cast<float2*>(row + c) = make_float2(first, second);
        }
      };
      for (int c = 2 * lane; c < R; c += 64)
        if (c < own || c >= own + u.width) pair(c, 0.0f, 0.0f);
#pragma unroll
      for (int i = 0; i < PAIRS; ++i) {
        const int c = 2 * (lane + 32 * i);
        if (c < u.width) pair(own + c, y[2 * i], y[2 * i + 1]);
      }
    } else {
      for (int c = lane; c < R; c += 32)
        if (c < own || c >= own + u.width) row[c] = hx_from_float<T>(0.0f);
#pragma unroll
      for (int i = 0; i < PAIRS; ++i) {
        const int c = 2 * (lane + 32 * i);
        if (c < u.width) row[own + c] = hx_from_float<T>(y[2 * i]);
        if (c + 1 < u.width) row[own + c + 1] = hx_from_float<T>(y[2 * i + 1]);
      }
    }
    return;
  }
  const int page = a.block_tables[static_cast<size_t>(table_row) * a.table_stride + position / a.page_size];
  if (page < 0 || page >= a.num_pages) {
    if (lane == 0 && a.status != nullptr) atomicOr(a.status, HX_FLAG_BAD_PAGE);
    return;
  }
  T* cache = u.kind == 1 ? a.k_cache : a.v_cache;
  const int slot = position % a.page_size;
  const int chunk = hx_cache_chunk(sizeof(T), R);
  auto place = [&](int d) {
    return cache + hx_cache_offset(page, u.head, slot, d, a.kv_heads, a.page_size, R, chunk);
  };
#pragma unroll
  for (int i = 0; i < PAIRS; ++i) {
    const int c = 2 * (lane + 32 * i);
    if constexpr (WIDE) {       // chunks are even and so are own and c
      if (c < u.width) {
        if constexpr (sizeof(T) == 2) {
          *reinterpret_cast<__nv_bfloat162*>(place(own + c)) = __floats2bfloat162_rn(y[2 * i], y[2 * i + 1]);
        } else {
          *reinterpret_cast<float2*>(place(own + c)) = make_float2(y[2 * i], y[2 * i + 1]);
        }
      }
    } else {
      if (c < u.width) *place(own + c) = hx_from_float<T>(y[2 * i]);
      if (c + 1 < u.width) *place(own + c + 1) = hx_from_float<T>(y[2 * i + 1]);
    }
  }
  // zeros behind the row's own coordinates (a page may have held anything before)
  const int used = u.kind == 2 ? a.vdim : a.maps * a.dim;
  if (u.kind == 2 || u.map == a.maps - 1)
    for (int d = used + lane; d < R; d += 32) *place(d) = hx_from_float<T>(0.0f);
}

// element c of a token's projection, sums rounded as the projection's own store would have
template <typename T>
__device__ __forceinline__ float projected_at(const FilteredHeadsArgs<T>& a, int token, int c) {
  if (a.accum != nullptr)
    return hx_to_float<T>(hx_from_float<T>(a.accum[static_cast<size_t>(token) * a.ld_accum + c]));
  return hx_to_float<T>(a.raw[static_cast<size_t>(token) * a.ld_raw + c]);
}

// Any sizes, one token per warp.
constexpr int ANY_PAIRS = 16;       // units up to 1,024 wide

template <typename T>
__global__ __launch_bounds__(128) void filtered_heads_kernel(const FilteredHeadsArgs<T> a, int units) {
  hx_pdl_prologue();
  const int token = blockIdx.x;
  const int index = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (index >= units) return;
  const int lane = threadIdx.x & 31;
  const Unit u = unit_of(a, index);
  const int request = a.token_request[token];
  const int start = a.request_start[request];
  const int place = token - start, reach = a.taps - 1;
  if (place > 0 && place < reach) return;        // the warp of the portion's first token does these
  const int table_row = a.request_slot[request];
  const int position = a.positions[token];
  const int count = a.request_start[request + 1] - start;
  float* state = a.state + static_cast<size_t>(table_row) * a.state_stride;
  const bool leads = place == 0;
  const int last = leads ? min(max(reach, 1), count) : 1;
  // an input: the portion's own row or, in front of it, the state's
  auto input = [&](int at, int c) {
    if (at >= 0) return projected_at(a, start + at, c) + (a.bias != nullptr ? a.bias[c] : 0.0f);
    return state[static_cast<size_t>(at + reach) * a.channels + c];
  };
  for (int t = 0; t < last; ++t) {
    float y[2 * ANY_PAIRS];
#pragma unroll
    for (int i = 0; i < 2 * ANY_PAIRS; ++i) {
      const int c = 2 * (lane + 32 * (i >> 1)) + (i & 1);
      y[i] = 0.0f;
      if (c < u.width) {
        const float* w = a.filter + static_cast<size_t>(u.column + c) * a.taps;
        for (int j = 0; j < a.taps; ++j)
          y[i] = fmaf(w[j], input(place + t - reach + j, u.column + c), y[i]);
      }
    }
    finish_unit<T, ANY_PAIRS, false>(a, u, token + t, position + t, table_row, y);
  }
  if (!leads) return;
  for (int c = lane; c < u.width; c += 32)
    for (int r = 0; r < reach; ++r)
      state[static_cast<size_t>(r) * a.channels + u.column + c] = input(count - reach + r, u.column + c);
}

// bfloat16 rows of even units and up to four taps: a warp walks `run` tokens and keeps the inputs of
// the tokens behind it.
template <int TAPS, int PAIRS>
__global__ __launch_bounds__(128) void filtered_heads_pairs_kernel(
    const FilteredHeadsArgs<__nv_bfloat16> a, int units) {
  constexpr int REACH = TAPS - 1;
  hx_pdl_trigger();
  const int first = blockIdx.x * a.run;
  const int last = min(first + a.run, a.tokens);
  const int index = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (index >= units) {
    hx_pdl_wait();      // a grid must not be seen complete before its predecessor is
    return;
  }
  const int lane = threadIdx.x & 31;
  const Unit u = unit_of(a, index);
  // weights, biases and the step's description do not depend on the kernel before
  float w[TAPS][2 * PAIRS], bias[2 * PAIRS];
#pragma unroll
  for (int i = 0; i < 2 * PAIRS; ++i) {
    const int c = 2 * (lane + 32 * (i >> 1)) + (i & 1);
    const bool live = c < u.width;
    bias[i] = live && a.bias != nullptr ? a.bias[u.column + c] : 0.0f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
      w[j][i] = live ? a.filter[static_cast<size_t>(u.column + c) * TAPS + j] : 0.0f;
  }
  int request = a.token_request[first];
  int start = a.request_start[request], end = a.request_start[request + 1];
  int slot = a.request_slot[request];
  hx_pdl_wait();
  auto input = [&](int token, float (&x)[2 * PAIRS]) {
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const int c = 2 * (lane + 32 * i);
      float2 v = make_float2(0.0f, 0.0f);
      if (c < u.width) {
        if (a.accum != nullptr) {
          const float2 s = *reinterpret_cast<const float2*>(
              a.accum + static_cast<size_t>(token) * a.ld_accum + u.column + c);
          v = __bfloat1622float2(__floats2bfloat162_rn(s.x, s.y));
        } else {
          v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(
              a.raw + static_cast<size_t>(token) * a.ld_raw + u.column + c));
        }
      }
      x[2 * i] = v.x + bias[2 * i];
      x[2 * i + 1] = v.y + bias[2 * i + 1];
    }
  };
  float x[TAPS][2 * PAIRS];       // inputs of tokens token - REACH .. token
#pragma unroll
  for (int j = 0; j < REACH; ++j)
    if (first - REACH + j >= start) input(first - REACH + j, x[j]);
#pragma unroll 1
  for (int token = first; token < last; ++token) {
    if (token >= end) {
      request = a.token_request[token];
      start = a.request_start[request];
      end = a.request_start[request + 1];
      slot = a.request_slot[request];
    }
    const int place = token - start;
    if (place == 0) {
      // the state stands for the tokens in front of the portion
      float* state = a.state + static_cast<size_t>(slot) * a.state_stride + u.column;
      const int count = end - start;
#pragma unroll
      for (int j = 0; j < REACH; ++j)
#pragma unroll
        for (int i = 0; i < PAIRS; ++i) {
          const int c = 2 * (lane + 32 * i);
          float2 v = make_float2(0.0f, 0.0f);
          if (c < u.width) v = *reinterpret_cast<const float2*>(state + static_cast<size_t>(j) * a.channels + c);
          x[j][2 * i] = v.x;
          x[j][2 * i + 1] = v.y;
        }
      // the portion's first tokens, whichever warps' runs they lie in; x walks with them
      const int behind = REACH > 0 ? min(REACH, count) : 1;
      float walk[TAPS][2 * PAIRS];
#pragma unroll
      for (int j = 0; j < REACH; ++j)
#pragma unroll
        for (int i = 0; i < 2 * PAIRS; ++i) walk[j][i] = x[j][i];
#pragma unroll 1
      for (int t = 0; t < behind; ++t) {
        input(start + t, walk[REACH]);
        float y[2 * PAIRS];
#pragma unroll
        for (int i = 0; i < 2 * PAIRS; ++i) {
          y[i] = 0.0f;
#pragma unroll
          for (int j = 0; j < TAPS; ++j) y[i] = fmaf(w[j][i], walk[j][i], y[i]);
        }
        finish_unit<__nv_bfloat16, PAIRS, true>(a, u, start + t, a.positions[start] + t, slot, y);
#pragma unroll
        for (int j = 0; j < REACH; ++j)
#pragma unroll
          for (int i = 0; i < 2 * PAIRS; ++i) walk[j][i] = walk[j + 1][i];
      }
      // the new state: the last REACH inputs up to the portion's end (`walk` holds them already
      // when the portion is no longer than that)
#pragma unroll
      for (int r = 0; r < REACH; ++r) {
        if (count > REACH) input(start + count - REACH + r, walk[r]);
#pragma unroll
        for (int i = 0; i < PAIRS; ++i) {
          const int c = 2 * (lane + 32 * i);
          if (c < u.width)
            *reinterpret_cast<float2*>(state + static_cast<size_t>(r) * a.channels + c) =
                make_float2(walk[r][2 * i], walk[r][2 * i + 1]);
        }
      }
    }
    input(token, x[REACH]);
    if (place >= REACH && !(REACH == 0 && place == 0)) {
      float y[2 * PAIRS];
#pragma unroll
      for (int i = 0; i < 2 * PAIRS; ++i) {
        y[i] = 0.0f;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) y[i] = fmaf(w[j][i], x[j][i], y[i]);
      }
      finish_unit<__nv_bfloat16, PAIRS, true>(a, u, token, a.positions[token], slot, y);
    }
#pragma unroll
    for (int j = 0; j < REACH; ++j)
#pragma unroll
      for (int i = 0; i < 2 * PAIRS; ++i) x[j][i] = x[j + 1][i];
  }
}

// bfloat16 rows whose heads are whole pieces of 8 channels, up to four taps.
__device__ __forceinline__ void unpack_piece(const uint4& packed, float (&x)[8]) {
  const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&packed);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 v = __bfloat1622float2(pairs[i]);
    x[2 * i] = v.x;
    x[2 * i + 1] = v.y;
  }
}

constexpr int EARLY_START_TOKENS = 16;

template <int TAPS>
__global__ __launch_bounds__(128) void filtered_heads_pieces_kernel(
    const FilteredHeadsArgs<__nv_bfloat16> a, int qk_lanes, int v_lanes) {
  constexpr int REACH = TAPS - 1;
  // few tokens: the attention kernel behind may find its keys while this one runs; with more, all of
  // its warps would leave their wait at once and stay in step, which costs more than the start saves
  if (a.tokens <= EARLY_START_TOKENS) hx_pdl_trigger();
  const int first = blockIdx.x * a.run;
  const int last = min(first + a.run, a.tokens);
  const int index = blockIdx.y * blockDim.x + threadIdx.x;     // among a token's lanes
  const int qk_units = (a.heads + a.kv_heads) * a.maps;
  const bool is_value = index >= qk_units * qk_lanes;
  const int own_lanes = is_value ? v_lanes : qk_lanes;
  const int within = is_value ? index - qk_units * qk_lanes : index;
  const int unit = within / own_lanes, piece = within - unit * own_lanes;
  // idle lanes (behind the last unit, or behind a unit's pieces) take part in the sums with zeros
  const bool live = is_value ? unit < a.kv_heads && 8 * piece < a.vdim : 8 * piece < a.dim;
  Unit u = unit_of(a, is_value ? (unit < a.kv_heads ? qk_units + unit : 0) : unit);
  const int c0 = u.column + 8 * piece;
  float w[TAPS][8], bias[8], weight[8];
  {
    float flat[8 * TAPS];
    const float4* source = reinterpret_cast<const float4*>(a.filter + static_cast<size_t>(c0) * TAPS);
#pragma unroll
    for (int v = 0; v < 2 * TAPS; ++v) {
      const float4 x = live ? source[v] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      flat[4 * v] = x.x; flat[4 * v + 1] = x.y; flat[4 * v + 2] = x.z; flat[4 * v + 3] = x.w;
    }
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < 8; ++i) w[j][i] = flat[i * TAPS + j];
  }
  const float* norm = u.kind == 0 ? a.q_norm : a.k_norm;
  const bool normed = u.kind != 2 && norm != nullptr;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    bias[i] = live && a.bias != nullptr ? a.bias[c0 + i] : 0.0f;
    weight[i] = live && normed ? norm[8 * piece + i] : 1.0f;
  }
  int request = a.token_request[first];
  int start = a.request_start[request], end = a.request_start[request + 1];
  int slot = a.request_slot[request];
  hx_pdl_wait();

  const int R = a.row_dim, half = a.rot >> 1, own = u.kind == 2 ? 0 : u.map * a.dim;
  const float over = 1.0f / static_cast<float>(u.width);
  auto finish = [&](int token, int position, float (&y)[8]) {
    if (a.q_norm != nullptr || a.k_norm != nullptr) {
      float sum = 0.0f;
#pragma unroll
      for (int i = 0; i < 8; ++i) sum = fmaf(y[i], y[i], sum);
#pragma unroll
      for (int offset = 1; offset < 32; offset <<= 1) {
        const float other = __shfl_xor_sync(0xffffffffu, sum, offset);
        if (offset < own_lanes) sum += other;
      }
      const float unit_scale = normed ? 1.0f / sqrtf(fmaf(sum, over, a.eps)) : 1.0f;
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] *= unit_scale * weight[i];
    }
    if (!live) return;
    if (u.kind != 2 && 8 * piece < a.rot) {
      if (position >= a.table_rows) {
        if (a.status != nullptr) atomicOr(a.status, HX_FLAG_BAD_POSITION);
        return;
      }
      const float* cosine = a.cosine + static_cast<size_t>(position) * half + 4 * piece;
      const float* sine = a.sine + static_cast<size_t>(position) * half + 4 * piece;
      float c[4], s[4];
      if ((a.rot & 7) == 0) {
        const float4 c4 = *reinterpret_cast<const float4*>(cosine), s4 = *reinterpret_cast<const float4*>(sine);
        c[0] = c4.x; c[1] = c4.y; c[2] = c4.z; c[3] = c4.w;
        s[0] = s4.x; s[1] = s4.y; s[2] = s4.z; s[3] = s4.w;
      } else {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const bool turns = 4 * piece + i < half;
          c[i] = turns ? cosine[i] : 1.0f;
          s[i] = turns ? sine[i] : 0.0f;
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float x = y[2 * i], z = y[2 * i + 1];
        y[2 * i] = x * c[i] - z * s[i];
        y[2 * i + 1] = z * c[i] + x * s[i];
      }
    }
    uint4 packed;
    __nv_bfloat162* pairs = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
    for (int i = 0; i < 4; ++i) pairs[i] = __floats2bfloat162_rn(y[2 * i], y[2 * i + 1]);
    const uint4 zeros = make_uint4(0u, 0u, 0u, 0u);
    if (u.kind == 0) {
      // the row's other pieces are zeros, dealt to the unit's lanes
      uint4* row = reinterpret_cast<uint4*>(a.out + static_cast<size_t>(token) * a.ld_out +
                                            (u.head * a.maps + u.map) * R);
      row[(own >> 3) + piece] = packed;
      const int mine = a.dim >> 3, from = own >> 3, others = (R >> 3) - mine;
      for (int p = piece; p < others; p += mine) row[p < from ? p : p + mine] = zeros;
      return;
    }
    const int page = a.block_tables[static_cast<size_t>(slot) * a.table_stride + position / a.page_size];
    if (page < 0 || page >= a.num_pages) {
      if (a.status != nullptr) atomicOr(a.status, HX_FLAG_BAD_PAGE);
      return;
    }
    __nv_bfloat16* cache = u.kind == 1 ? a.k_cache : a.v_cache;
    const int place = position % a.page_size;
    auto at = [&](int d) {
      return reinterpret_cast<uint4*>(cache + hx_cache_offset(page, u.head, place, d, a.kv_heads, a.page_size, R, 8));
    };
    *at(own + 8 * piece) = packed;
    const int used = u.kind == 2 ? a.vdim : a.maps * a.dim;
    if (u.kind == 2 || u.map == a.maps - 1)
      for (int d = used + 8 * piece; d < R; d += u.width) *at(d) = zeros;
  };
  auto packed_input = [&](int token) {
    if (!live) return make_uint4(0u, 0u, 0u, 0u);
    if (a.accum == nullptr)
      return *reinterpret_cast<const uint4*>(a.raw + static_cast<size_t>(token) * a.ld_raw + c0);
    const float4* source =
        reinterpret_cast<const float4*>(a.accum + static_cast<size_t>(token) * a.ld_accum + c0);
    const float4 lo = source[0], hi = source[1];
    uint4 packed;
    __nv_bfloat162* pairs = reinterpret_cast<__nv_bfloat162*>(&packed);
    pairs[0] = __floats2bfloat162_rn(lo.x, lo.y);
    pairs[1] = __floats2bfloat162_rn(lo.z, lo.w);
    pairs[2] = __floats2bfloat162_rn(hi.x, hi.y);
    pairs[3] = __floats2bfloat162_rn(hi.z, hi.w);
    return packed;
  };
  // inside a portion the bias passes the filter as a constant
  float inside[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    float sum = 0.0f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) sum += w[j][i];
    inside[i] = sum * bias[i];
  }
  uint4 rows[TAPS];      // inputs of tokens token - REACH .. token, without the bias
#pragma unroll
  for (int j = 0; j < REACH; ++j)
    rows[j] = first - REACH + j >= start ? packed_input(first - REACH + j) : make_uint4(0u, 0u, 0u, 0u);
  uint4 ahead = packed_input(first);
#pragma unroll 1
  for (int token = first; token < last; ++token) {
    rows[REACH] = ahead;
    if (token + 1 < last) ahead = packed_input(token + 1);
    if (token >= end) {
      request = a.token_request[token];
      start = a.request_start[request];
      end = a.request_start[request + 1];
      slot = a.request_slot[request];
    }
    const int place = token - start;
    if (place >= REACH && place > 0) {
      float y[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] = inside[i];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        float x[8];
        unpack_piece(rows[j], x);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = fmaf(w[j][i], x[i], y[i]);
      }
      finish(token, a.positions[token], y);
    } else if (place == 0) {
      const int count = end - start, position = a.positions[token];
      float* state = a.state + static_cast<size_t>(slot) * a.state_stride + c0;
      // an input with its bias: the portion's own, or in front of it the state's
      auto load = [&](int at, float (&x)[8]) {
        if (at >= 0) {
          unpack_piece(packed_input(start + at), x);
#pragma unroll
          for (int i = 0; i < 8; ++i) x[i] += bias[i];
        } else {
#pragma unroll
          for (int i = 0; i < 8; i += 4) {
            const float4 v = live ? *reinterpret_cast<const float4*>(
                                        state + static_cast<size_t>(at + REACH) * a.channels + i)
                                  : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            x[i] = v.x; x[i + 1] = v.y; x[i + 2] = v.z; x[i + 3] = v.w;
          }
        }
      };
      const int behind = REACH > 0 ? min(REACH, count) : 1;
#pragma unroll 1
      for (int t = 0; t < behind; ++t) {
        float y[8] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
          float x[8];
          load(t - REACH + j, x);
#pragma unroll
          for (int i = 0; i < 8; ++i) y[i] = fmaf(w[j][i], x[i], y[i]);
        }
        finish(start + t, position + t, y);
      }
      // the new state: the last REACH inputs up to the portion's end (ascending rows read ahead of
      // where they write)
#pragma unroll
      for (int r = 0; r < REACH; ++r) {
        float x[8];
        load(count - REACH + r, x);
        if (live) {
          float* target = state + static_cast<size_t>(r) * a.channels;
          *reinterpret_cast<float4*>(target) = make_float4(x[0], x[1], x[2], x[3]);
          *reinterpret_cast<float4*>(target + 4) = make_float4(x[4], x[5], x[6], x[7]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < REACH; ++j) rows[j] = rows[j + 1];
  }
}

bool heads_pieces_apply(const FilteredHeadsArgs<__nv_bfloat16>& a) {
  auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  return a.taps <= 4 && a.dim % 8 == 0 && a.dim <= 256 && a.row_dim % 8 == 0 && a.ld_out % 8 == 0 &&
         aligned(a.out) && aligned(a.filter) && (a.taps == 1 || aligned(a.state)) &&
         a.state_stride % 4 == 0 && (a.rot == 0 || (aligned(a.cosine) && aligned(a.sine))) &&
         (a.accum != nullptr ? a.ld_accum % 4 == 0 && aligned(a.accum) : a.ld_raw % 8 == 0 && aligned(a.raw)) &&
         (a.kv_heads == 0 ||
          (a.vdim % 8 == 0 && a.vdim <= 256 && aligned(a.k_cache) && aligned(a.v_cache)));
}

bool heads_pairs_apply(const FilteredHeadsArgs<__nv_bfloat16>& a) {
  auto aligned = [](const void* p, uintptr_t to) { return (reinterpret_cast<uintptr_t>(p) & (to - 1)) == 0; };
  return a.taps <= 4 && a.dim % 2 == 0 && a.vdim % 2 == 0 && a.dim <= 256 && a.vdim <= 256 &&
         a.row_dim % 2 == 0 && a.ld_out % 2 == 0 && aligned(a.out, 4) && aligned(a.state, 8) &&
         a.state_stride % 2 == 0 &&
         (a.accum != nullptr ? a.ld_accum % 2 == 0 && aligned(a.accum, 8)
                             : a.ld_raw % 2 == 0 && aligned(a.raw, 4)) &&
         (a.kv_heads == 0 || (aligned(a.k_cache, 4) && aligned(a.v_cache, 4)));
}

template <int TAPS>
void launch_heads_pairs(const FilteredHeadsArgs<__nv_bfloat16>& a, dim3 grid, int units, int widest,
                        cudaStream_t stream) {
  if (widest <= 64) {
    hx_launch(filtered_heads_pairs_kernel<TAPS, 1>, grid, 128, 0, stream, a, units);
  } else if (widest <= 128) {
    hx_launch(filtered_heads_pairs_kernel<TAPS, 2>, grid, 128, 0, stream, a, units);
  } else {
    hx_launch(filtered_heads_pairs_kernel<TAPS, 4>, grid, 128, 0, stream, a, units);
  }
}

template <typename T>
void launch_filtered_heads(FilteredHeadsArgs<T> a, cudaStream_t stream) {
  const int units = (a.heads + a.kv_heads) * a.maps + a.kv_heads;
  if constexpr (sizeof(T) == 2) {
    if (heads_pieces_apply(a)) {
      auto lanes = [](int width) {
        int n = 1;
        while (8 * n < width) n *= 2;
        return n;
      };
      a.run = a.tokens >= 1024 ? 8 : (a.tokens >= 256 ? 4 : 1);
      const int qk_lanes = lanes(a.dim), v_lanes = lanes(a.vdim);
      const int all = (a.heads + a.kv_heads) * a.maps * qk_lanes + a.kv_heads * v_lanes;
      const dim3 grid((a.tokens + a.run - 1) / a.run, (all + 127) / 128);
      switch (a.taps) {
        case 1: hx_launch(filtered_heads_pieces_kernel<1>, grid, 128, 0, stream, a, qk_lanes, v_lanes); return;
        case 2: hx_launch(filtered_heads_pieces_kernel<2>, grid, 128, 0, stream, a, qk_lanes, v_lanes); return;
        case 3: hx_launch(filtered_heads_pieces_kernel<3>, grid, 128, 0, stream, a, qk_lanes, v_lanes); return;
        default: hx_launch(filtered_heads_pieces_kernel<4>, grid, 128, 0, stream, a, qk_lanes, v_lanes); return;
      }
    }
    if (heads_pairs_apply(a)) {
      a.run = a.tokens >= 1024 ? 8 : (a.tokens >= 256 ? 4 : 1);
      const dim3 grid((a.tokens + a.run - 1) / a.run, (units + 3) / 4);
      const int widest = a.kv_heads > 0 ? max(a.dim, a.vdim) : a.dim;
      switch (a.taps) {
        case 1: launch_heads_pairs<1>(a, grid, units, widest, stream); return;
        case 2: launch_heads_pairs<2>(a, grid, units, widest, stream); return;
        case 3: launch_heads_pairs<3>(a, grid, units, widest, stream); return;
        default: launch_heads_pairs<4>(a, grid, units, widest, stream); return;
      }
    }
  }
  hx_launch(filtered_heads_kernel<T>, dim3(a.tokens, (units + 3) / 4), 128, 0, stream, a, units);
}

// ------------------------------------------------------------------- difference of maps

template <typename T>
struct MapDifferenceArgs {
  const T* context;         // [tokens, ld_context]: 2 * heads rows of row_dim
  int ld_context;
  const T* gate;            // [tokens, ld_gate], or
  int ld_gate;
  const float* gate_sums;   // float32 sums [tokens, ld_sums] (null: `gate`), rounded when read
  int ld_sums;
  float lambda, scale, eps;
  T* out;                   // [tokens, ld_out]: heads * vdim
  int ld_out;
  float* clear;             // accumulator rows to zero: [tokens, ld_clear], clear_width columns; or null
  int ld_clear, clear_width;
  int heads, vdim, row_dim;
};

constexpr int DIFFERENCE_WARPS = 4;

// grid (tokens, ceil(heads / DIFFERENCE_WARPS)).  HELD numbers a lane are kept between the passes.  Any
// sizes.
template <typename T, int HELD>
__global__ __launch_bounds__(DIFFERENCE_WARPS * 32) void map_difference_kernel(const MapDifferenceArgs<T> a) {
  hx_pdl_prologue();
  const size_t token = blockIdx.x;
  const int head = blockIdx.y * DIFFERENCE_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (head >= a.heads) return;
  const T* first = a.context + token * a.ld_context + static_cast<size_t>(2 * head) * a.row_dim;
  const T* second = first + a.row_dim;
  auto difference = [&](int c) {
    return hx_to_float<T>(first[c]) - a.lambda * hx_to_float<T>(second[c]);
  };
  float o[HELD], g[HELD];
  float sum = 0.0f;
  auto gate_at = [&](int c) {
    const int column = head * a.vdim + c;
    if (a.gate_sums != nullptr) return hx_to_float<T>(hx_from_float<T>(a.gate_sums[token * a.ld_sums + column]));
    return hx_to_float<T>(a.gate[token * a.ld_gate + column]);
  };
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int c = lane + 32 * i;
    o[i] = c < a.vdim ? difference(c) : 0.0f;
    g[i] = c < a.vdim ? gate_at(c) : 0.0f;
  }
#pragma unroll
  for (int i = 0; i < HELD; ++i) sum = fmaf(o[i], o[i], sum);
  for (int c = lane + 32 * HELD; c < a.vdim; c += 32) {
    const float v = difference(c);
    sum = fmaf(v, v, sum);
  }
  const float unit = a.scale / sqrtf(warp_sum(sum) / static_cast<float>(a.vdim) + a.eps);
  T* out = a.out + token * a.ld_out + head * a.vdim;
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int c = lane + 32 * i;
    if (c < a.vdim) out[c] = hx_from_float<T>(o[i] * unit * hx_sigmoid(g[i]));
  }
  for (int c = lane + 32 * HELD; c < a.vdim; c += 32)
    out[c] = hx_from_float<T>(difference(c) * unit * hx_sigmoid(gate_at(c)));
  if (a.clear != nullptr) {
    // a head's warp clears its share of the row: the gate's columns, which lie at the row's end, are
    // its own (it has read them); of the rest an equal part
    float* row = a.clear + token * a.ld_clear;
    const int gates = a.heads * a.vdim, rest = a.clear_width - gates;
    const int from = static_cast<int>(static_cast<long long>(rest) * head / a.heads);
    const int to = static_cast<int>(static_cast<long long>(rest) * (head + 1) / a.heads);
    for (int c = from + lane; c < to; c += 32) row[c] = 0.0f;
    for (int c = lane; c < a.vdim; c += 32) row[rest + head * a.vdim + c] = 0.0f;
  }
}

// Four numbers at a time, for heads of up to 256 values in whole pieces of four.
__device__ __forceinline__ float4 load_quad(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load_quad(const __nv_bfloat16* p) {
  const uint2 packed = *reinterpret_cast<const uint2*>(p);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&packed.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&packed.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void store_quad(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store_quad(__nv_bfloat16* p, float4 v) {
  uint2 packed;
  *reinterpret_cast<__nv_bfloat162*>(&packed.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&packed.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = packed;
}
// results stored in bfloat16 take the hardware exponential
template <typename T> __device__ __forceinline__ float gate_factor(float x) {
  if constexpr (sizeof(T) == 4) return hx_sigmoid(x);
  return __fdividef(1.0f, 1.0f + __expf(-hx_to_float<T>(hx_from_float<T>(x))));
}

template <typename T>
__global__ __launch_bounds__(DIFFERENCE_WARPS * 32) void map_difference_quads_kernel(const MapDifferenceArgs<T> a) {
  constexpr int HELD = 2;
  hx_pdl_prologue();
  const size_t token = blockIdx.x;
  const int head = blockIdx.y * DIFFERENCE_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (head >= a.heads) return;
  const T* first = a.context + token * a.ld_context + static_cast<size_t>(2 * head) * a.row_dim;
  const int quads = a.vdim >> 2, column = head * a.vdim;
  const float4 zeros = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  float4 x[HELD], y[HELD], g[HELD];
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int q = lane + 32 * i;
    x[i] = y[i] = g[i] = zeros;
    if (q < quads) {
      x[i] = load_quad(first + 4 * q);
      y[i] = load_quad(first + a.row_dim + 4 * q);
      g[i] = a.gate_sums != nullptr ? load_quad(a.gate_sums + token * a.ld_sums + column + 4 * q)
                                    : load_quad(a.gate + token * a.ld_gate + column + 4 * q);
    }
  }
  float sum = 0.0f;
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    x[i].x -= a.lambda * y[i].x; x[i].y -= a.lambda * y[i].y;
    x[i].z -= a.lambda * y[i].z; x[i].w -= a.lambda * y[i].w;
    sum = fmaf(x[i].x, x[i].x, sum); sum = fmaf(x[i].y, x[i].y, sum);
    sum = fmaf(x[i].z, x[i].z, sum); sum = fmaf(x[i].w, x[i].w, sum);
  }
  const float unit = a.scale / sqrtf(warp_sum(sum) / static_cast<float>(a.vdim) + a.eps);
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int q = lane + 32 * i;
    if (q < quads)
      store_quad(a.out + token * a.ld_out + column + 4 * q,
                 make_float4(x[i].x * unit * gate_factor<T>(g[i].x), x[i].y * unit * gate_factor<T>(g[i].y),
                             x[i].z * unit * gate_factor<T>(g[i].z), x[i].w * unit * gate_factor<T>(g[i].w)));
  }
  if (a.clear != nullptr) {
    // see map_difference_kernel: the head's own gate columns, and its share of the rest
    float* row = a.clear + token * a.ld_clear;
    const int rest = (a.clear_width - a.heads * a.vdim) >> 2;
    const int from = static_cast<int>(static_cast<long long>(rest) * head / a.heads);
    const int to = static_cast<int>(static_cast<long long>(rest) * (head + 1) / a.heads);
    for (int q = from + lane; q < to; q += 32) store_quad(row + 4 * q, zeros);
    for (int q = lane; q < quads; q += 32) store_quad(row + 4 * rest + column + 4 * q, zeros);
  }
}

template <typename T>
void launch_map_difference(const MapDifferenceArgs<T>& a, int tokens, cudaStream_t stream) {
  const dim3 grid(tokens, (a.heads + DIFFERENCE_WARPS - 1) / DIFFERENCE_WARPS);
  auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  if (a.vdim % 4 == 0 && a.vdim <= 256 && a.row_dim % 4 == 0 && a.ld_context % 4 == 0 && a.ld_out % 4 == 0 &&
      (a.gate_sums != nullptr ? a.ld_sums : a.ld_gate) % 4 == 0 && aligned(a.context) && aligned(a.out) &&
      aligned(a.gate_sums) && (reinterpret_cast<uintptr_t>(a.gate) & 7) == 0 && (sizeof(T) == 2 || aligned(a.gate)) &&
      (a.clear == nullptr || (a.ld_clear % 4 == 0 && a.clear_width % 4 == 0 && aligned(a.clear)))) {
    hx_launch(map_difference_quads_kernel<T>, grid, DIFFERENCE_WARPS * 32, 0, stream, a);
  } else if (a.vdim <= 128) {
    hx_launch(map_difference_kernel<T, 4>, grid, DIFFERENCE_WARPS * 32, 0, stream, a);
  } else {
    hx_launch(map_difference_kernel<T, 8>, grid, DIFFERENCE_WARPS * 32, 0, stream, a);
  }
}

}  // namespace

// See the head of this file.  raw [tokens, ld_raw] in `dtype` or accum float32 sums is given, the other
// null; the columns behind the filtered ones are not touched.  kv_heads 0 (a layer that uses another
// layer's keys and values): the rows hold queries only.  state may be null with one tap; bias,
// q_norm and k_norm may be null; rot 0: no rotation.
HX_API int hx_filtered_heads(const void* raw, int ld_raw, const float* accum, int ld_accum, int dtype,
                             const float* bias, const float* filter, int taps, float* state,
                             long long state_stride, const float* q_norm, const float* k_norm, float eps,
                             const float* cosine, const float* sine, int rot, int table_rows, void* out,
                             int ld_out, void* k_cache, void* v_cache, const int* positions,
                             const int* token_request, const int* request_slot,
                             const int* request_start, const int* block_tables, int table_stride,
                             int tokens, int heads, int kv_heads, int maps, int dim, int vdim,
                             int row_dim, int page_size, int num_pages, int* status,
                             cudaStream_t stream) {
  HX_REQUIRE(tokens >= 0 && heads > 0 && kv_heads >= 0 && maps > 0 && dim > 0 && vdim > 0 &&
                 row_dim >= maps * dim && (kv_heads == 0 || row_dim >= vdim),
             "hx_filtered_heads: bad sizes");
  HX_REQUIRE(dim <= 64 * ANY_PAIRS && (kv_heads == 0 || vdim <= 64 * ANY_PAIRS),
             "hx_filtered_heads: heads wider than %d", 64 * ANY_PAIRS);
  const int channels = (heads + kv_heads) * maps * dim + kv_heads * vdim;
  HX_REQUIRE((raw != nullptr) != (accum != nullptr),
             "hx_filtered_heads: give the projected rows or their sums");
  HX_REQUIRE((raw == nullptr || ld_raw >= channels) && (accum == nullptr || ld_accum >= channels) &&
                 ld_out >= heads * maps * row_dim, "hx_filtered_heads: row strides too small");
  HX_REQUIRE(filter != nullptr && taps >= 1 && (taps == 1 || (state != nullptr &&
                 state_stride >= static_cast<long long>(taps - 1) * channels)),
             "hx_filtered_heads: filter or state missing");
  HX_REQUIRE((q_norm == nullptr && k_norm == nullptr) || eps > 0.0f, "hx_filtered_heads: eps must be positive");
  HX_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= dim &&
                 (rot == 0 || (cosine != nullptr && sine != nullptr && table_rows > 0)),
             "hx_filtered_heads: rotation over %d of %d coordinates", rot, dim);
  HX_REQUIRE(kv_heads == 0 || (k_cache != nullptr && v_cache != nullptr && block_tables != nullptr &&
                               page_size > 0 && num_pages > 0 && table_stride > 0),
             "hx_filtered_heads: cache arguments missing");
  const int units = (heads + kv_heads) * maps + kv_heads;
  HX_REQUIRE((units + 3) / 4 <= 65535, "hx_filtered_heads: too many heads");
  if (tokens == 0) return HX_OK;
  if (dtype == HX_F32) {
    launch_filtered_heads(
        FilteredHeadsArgs<float>{static_cast<const float*>(raw), ld_raw, accum, ld_accum, bias, filter,
                                 state, state_stride, taps, channels, q_norm, k_norm, eps, cosine, sine,
                                 rot, table_rows, static_cast<float*>(out), ld_out,
                                 static_cast<float*>(k_cache), static_cast<float*>(v_cache), positions,
                                 token_request, request_slot, request_start, block_tables, table_stride,
                                 tokens, 1, heads, kv_heads, maps, dim, vdim, row_dim, page_size,
                                 num_pages, status},
        stream);
  } else if (dtype == HX_BF16) {
    launch_filtered_heads(
        FilteredHeadsArgs<__nv_bfloat16>{
            static_cast<const __nv_bfloat16*>(raw), ld_raw, accum, ld_accum, bias, filter, state,
            state_stride, taps, channels, q_norm, k_norm, eps, cosine, sine, rot, table_rows,
            static_cast<__nv_bfloat16*>(out), ld_out, static_cast<__nv_bfloat16*>(k_cache),
            static_cast<__nv_bfloat16*>(v_cache), positions, token_request, request_slot, request_start,
            block_tables, table_stride, tokens, 1, heads, kv_heads, maps, dim, vdim, row_dim, page_size,
            num_pages, status},
        stream);
  } else {
    HX_REQUIRE(false, "hx_filtered_heads: unknown dtype %d", dtype);
  }
  HX_CHECK_LAUNCH("hx_filtered_heads");
  return HX_OK;
}

// context [tokens, ld_context] in `dtype`: per head two rows of row_dim (map 1, map 2), the first vdim
// coordinates of each used.  gate in `dtype` or gate_sums float32 (the other null), [tokens, heads *
// vdim].  out [tokens, heads * vdim] in `dtype`.  clear (may be null): accumulator rows of clear_width
// columns to zero, of which gate_sums must be the last heads * vdim when it is given.
HX_API int hx_map_difference(const void* context, int ld_context, const void* gate, int ld_gate,
                             const float* gate_sums, int ld_sums, int dtype, float lambda, float scale,
                             float eps, void* out, int ld_out, float* clear, int ld_clear,
                             int clear_width, int tokens, int heads, int vdim, int row_dim,
                             cudaStream_t stream) {
  HX_REQUIRE(tokens >= 0 && heads > 0 && heads <= 65535 * DIFFERENCE_WARPS && vdim > 0 &&
                 row_dim >= vdim && eps > 0.0f && ld_context >= 2 * heads * row_dim &&
                 ld_out >= heads * vdim, "hx_map_difference: bad sizes");
  HX_REQUIRE((gate != nullptr) != (gate_sums != nullptr), "hx_map_difference: give the gate or its sums");
  HX_REQUIRE((gate == nullptr || ld_gate >= heads * vdim) && (gate_sums == nullptr || ld_sums >= heads * vdim),
             "hx_map_difference: gate stride too small");
  HX_REQUIRE(clear == nullptr || (clear_width >= heads * vdim && ld_clear >= clear_width &&
                                  (gate_sums == nullptr || gate_sums == clear + (clear_width - heads * vdim))),
             "hx_map_difference: bad accumulator");
  if (tokens == 0) return HX_OK;
  if (dtype == HX_F32) {
    launch_map_difference(
        MapDifferenceArgs<float>{static_cast<const float*>(context), ld_context,
                                 static_cast<const float*>(gate), ld_gate, gate_sums, ld_sums, lambda,
                                 scale, eps, static_cast<float*>(out), ld_out, clear, ld_clear,
                                 clear_width, heads, vdim, row_dim},
        tokens, stream);
  } else if (dtype == HX_BF16) {
    launch_map_difference(
        MapDifferenceArgs<__nv_bfloat16>{
            static_cast<const __nv_bfloat16*>(context), ld_context,
            static_cast<const __nv_bfloat16*>(gate), ld_gate, gate_sums, ld_sums, lambda, scale, eps,
            static_cast<__nv_bfloat16*>(out), ld_out, clear, ld_clear, clear_width, heads, vdim, row_dim},
        tokens, stream);
  } else {
    HX_REQUIRE(false, "hx_map_difference: unknown dtype %d", dtype);
  }
  HX_CHECK_LAUNCH("hx_map_difference");
  return HX_OK;
}
