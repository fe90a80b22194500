// A feed-forward that routes every token to `top` of E experts.
//
//  gb_op_moe_route     per token: the `top` largest router logits (ties: the lower index), their
//                      sigmoids as weights (not renormalised), and the sigmoid of the shared expert's
//                      gate logit; all in 32-bit
//  gb_op_moe_route_grouped  the same choice for routers with softmax (or sigmoid) scores, a correction added to
//                      the scores for the choice only, experts in groups of which only the best are open, and
//                      trailing "identity" outputs that stand for experts returning their input
//  gb_op_moe_sort      (token, choice) pairs ordered by expert: offsets[E + 1], the pair behind every
//                      row, the row of every pair
//  gb_op_moe_gather    rows[row] = weight * h[token]: the weight multiplies the expert's INPUT
//  gb_op_moe_dispatch  the grouped choice, the order and the gathered rows together (one kernel for a step of few tokens)
//  gb_op_moe_experts   per expert, over its rows: act = glu(rows W_gate^T, rows W_up^T) with clamps, or act =
//                      function(rows W_up^T) for experts without a gate, or out = rows W_down^T (32-bit)
//  gb_op_moe_combine   y[token] = sum over its choices of out[row] (+ gate * shared[token])
//  gb_op_moe_combine_weighted  y[token] (+)= sum over its choices of weight * out[row], where the weight multiplies
//                      the expert's OUTPUT; a choice beyond the real experts contributes weight * h[token]; optionally
//                      + shared[token], and the norm in front of the next sublayer taken of the new rows
//
// A row's result does not depend on which rows share its tile (one accumulator per output walking k
// upwards), so the order in which pairs land inside an expert's range does not matter.
#include "hybrid.cuh"

namespace {

constexpr int MOE_MAX_EXPERTS = 1024;

// one warp per token: lane l looks after experts l, l + 32, ... (a bit per expert it has given away)
__global__ void moe_route_kernel(const float* logits, long long ld, int n, int E, int top, int shared_col, int* idx,
                                 float* weight, float* shared_gate) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (t >= n) return;
  const float* z = logits + (size_t)t * ld;
  unsigned taken = 0;
  for (int k = 0; k < top; ++k) {
    float bv = -INFINITY;
    int be = 0x7fffffff;
    for (int i = 0, e = lane; e < E; ++i, e += 32) {
      if ((taken >> i) & 1u) continue;
      const float v = z[e];
      if (v > bv || be == 0x7fffffff) { bv = v; be = e; }   // (ascending e: a tie keeps the lower index)
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (oe != 0x7fffffff && (be == 0x7fffffff || ov > bv || (ov == bv && oe < be))) { bv = ov; be = oe; }
    }
    if ((be & 31) == lane) taken |= 1u << (be >> 5);
    if (lane == 0) {
      idx[(size_t)t * top + k] = be;
      weight[(size_t)t * top + k] = hy_sigmoid(bv);
    }
  }
  if (shared_gate && lane == 0) shared_gate[t] = hy_sigmoid(z[shared_col]);
}

// A router's rule.  scores: 0 sigmoid(z), 1 softmax(z) over all `n_out` router outputs, 2 the logits z themselves.
// `normalise`: 0 a chosen output's weight is its score, 1 the score divided by the sum of the chosen scores, 2 the
// softmax over the chosen scores alone.  The choice is made on
// score + correction; with `groups` > 1 the outputs form that many equal groups of neighbours, a group's mark is
// its largest choice score (or, with `mark_two`, the sum of its two largest), and only outputs of the `keep` best groups
// can be chosen.  The weight of a chosen output is its score without the correction, not renormalised, times
// `weight_scale`.  Ties go to the lower index.
struct RouteParams {
  const float* logits; long long ld;
  // instead of logits: the partial tiles [splits][n * n_out] of the product that makes them (+ bias)
  const float* part; int splits; const float* part_bias; long long part_stride;
  int n, n_out, top, scores, groups, keep, normalise, mark_two;
  const float* correction;
  float weight_scale;
};

// A 32-bit number whose order as an unsigned integer is the order of floats (no NaNs).
__device__ __forceinline__ unsigned ordered(float v) {
  const unsigned b = __float_as_uint(v);
  return b & 0x80000000u ? ~b : b | 0x80000000u;
}

// At most 32 router outputs, sigmoid scores or logits, weights as they are: a lane an output, maxima by one reduction over the
// warp and ties by the lowest lane.  The same choices and weights as below.
__device__ __forceinline__ void route_token_32(const RouteParams& p, float z, int lane, int* idx, float* weight) {
  const bool in = lane < p.n_out;
  const float s = p.scores == 0 ? hy_sigmoid(z) : z;
  const float c = s + (in && p.correction ? p.correction[lane] : 0.f);
  bool open = in;
  if (p.groups > 1 && p.keep < p.groups) {
    const int gs = p.n_out / p.groups;
    const int g = lane < p.groups ? lane : 0;             // lane g marks group g
    float b = -INFINITY, second = -INFINITY;
    for (int e = 0; e < gs; ++e) {
      const float v = __shfl_sync(0xffffffffu, c, g * gs + e);
      second = fmaxf(second, fminf(b, v));
      b = fmaxf(b, v);
    }
    const unsigned mark = lane < p.groups ? max(ordered(p.mark_two && gs > 1 ? b + second : b), 1u) : 0u;
    unsigned kept = 0;
    for (int k = 0; k < p.keep; ++k) {
      const unsigned mine = (kept >> lane) & 1u ? 0u : mark;
      const unsigned top = __reduce_max_sync(0xffffffffu, mine);
      kept |= 1u << (__ffs(__ballot_sync(0xffffffffu, mine == top)) - 1);
    }
    open = in && ((kept >> (lane / gs)) & 1u);
  }
  unsigned key = open ? max(ordered(c), 2u) : in ? 1u : 0u;
  for (int k = 0; k < p.top; ++k) {
    const unsigned top = __reduce_max_sync(0xffffffffu, key);
    const int e = __ffs(__ballot_sync(0xffffffffu, key == top)) - 1;
    if (lane == e) {
      idx[k] = e;
      weight[k] = s * p.weight_scale;
      key = 1u;                                            // taken
    }
  }
}

// One warp, one token; s, c [n_out] and mark [groups] are the warp's own shared memory.  Writes top choices and weights.
__device__ __forceinline__ void route_token(const RouteParams& p, int t, float* s, float* c, float* mark, int lane, int* idx,
                                            float* weight) {
  const int n_out = p.n_out, top = p.top;
  auto logit = [&](int e) {
    if (!p.part) return p.logits[(size_t)t * p.ld + e];
    float z;
    const size_t at = (size_t)t * n_out + e;
    sum_partials<1>(p.part, p.splits, (size_t)p.part_stride, &at, &z);
    return p.part_bias ? z + p.part_bias[e] : z;
  };
  if (n_out <= 32 && p.scores != 1 && !p.normalise) {
    route_token_32(p, lane < n_out ? logit(lane) : 0.f, lane, idx, weight);
    return;
  }
  for (int e = lane; e < n_out; e += 32) {
    const float z = logit(e);
    s[e] = p.scores == 0 ? hy_sigmoid(z) : z;
  }
  if (p.scores == 1) {                                    // (every lane its own entries: no barrier in between)
    float mx = -INFINITY;
    for (int e = lane; e < n_out; e += 32) mx = fmaxf(mx, s[e]);
    mx = warp_max(mx);
    float sum = 0.f;
    for (int e = lane; e < n_out; e += 32) {
      const float v = expf(s[e] - mx);
      s[e] = v;
      sum += v;
    }
    sum = warp_sum(sum);
    for (int e = lane; e < n_out; e += 32) s[e] = s[e] / sum;
  }
  for (int e = lane; e < n_out; e += 32) c[e] = s[e] + (p.correction ? p.correction[e] : 0.f);
  __syncwarp();
  const int gs = n_out / p.groups;
  if (p.groups > 1 && p.keep < p.groups) {
    for (int g = lane; g < p.groups; g += 32) {
      float b = -INFINITY, second = -INFINITY;
      for (int e = g * gs; e < (g + 1) * gs; ++e) {
        second = fmaxf(second, fminf(b, c[e]));
        b = fmaxf(b, c[e]);
      }
      mark[g] = p.mark_two && gs > 1 ? b + second : b;
    }
    __syncwarp();
    // the `keep` best groups stay open: the mark of a group that is picked becomes +infinity, which no score
    // reaches, so that the pass below reads one flag per group
    for (int k = 0; k < p.keep; ++k) {
      float bv = -INFINITY;
      int bg = 0x7fffffff;
      for (int g = lane; g < p.groups; g += 32) {
        const float v = mark[g];
        if (v != INFINITY && (bg == 0x7fffffff || v > bv)) { bv = v; bg = g; }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
        const int og = __shfl_xor_sync(0xffffffffu, bg, o);
        if (og != 0x7fffffff && (bg == 0x7fffffff || ov > bv || (ov == bv && og < bg))) { bv = ov; bg = og; }
      }
      if (lane == 0 && bg != 0x7fffffff) mark[bg] = INFINITY;
      __syncwarp();
    }
    for (int e = lane; e < n_out; e += 32)
      if (mark[e / gs] != INFINITY) c[e] = -INFINITY;     // (a closed output; an open one keeps its own score)
    __syncwarp();
  }
  for (int k = 0; k < top; ++k) {
    float bv = -INFINITY;
    int be = 0x7fffffff;
    for (int e = lane; e < n_out; e += 32) {
      const float v = c[e];
      if (v != -INFINITY || be == 0x7fffffff)
        if (be == 0x7fffffff || v > bv) { bv = v; be = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (oe != 0x7fffffff && (be == 0x7fffffff || ov > bv || (ov == bv && oe < be))) { bv = ov; be = oe; }
    }
    if (lane == 0) {
      idx[k] = be;
      weight[k] = p.normalise ? s[be] : s[be] * p.weight_scale;
      c[be] = -INFINITY;                                   // taken
    }
    __syncwarp();
  }
  if (p.normalise && lane == 0) {
    float sum = 0.f;
    if (p.normalise == 2) {
      const float mx = weight[0];                           // (the first choice has the largest score)
      for (int k = 0; k < top; ++k) {
        weight[k] = expf(weight[k] - mx);
        sum += weight[k];
      }
    } else {
      for (int k = 0; k < top; ++k) sum += weight[k];
    }
    for (int k = 0; k < top; ++k) weight[k] = weight[k] / sum * p.weight_scale;
  }
}

// one warp per token
__global__ void moe_route_grouped_kernel(RouteParams p, int* idx, float* weight) {
  extern __shared__ float route_sm[];                    // per warp: scores [n_out], choice scores [n_out], group marks
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t = blockIdx.x * (blockDim.x >> 5) + warp;
  if (t >= p.n) return;
  float* s = route_sm + (size_t)warp * (2 * p.n_out + p.groups);
  route_token(p, t, s, s + p.n_out, s + 2 * p.n_out, lane, idx + (size_t)t * p.top, weight + (size_t)t * p.top);
}

// A row copied in pieces of 16 bytes by the whole block.
__device__ __forceinline__ void copy_row16(const void* src, void* dst, int pieces) {
  for (int i = threadIdx.x; i < pieces; i += blockDim.x) static_cast<uint4*>(dst)[i] = static_cast<const uint4*>(src)[i];
}

// A step of few tokens: the choice, the pairs in the experts' order and the gathered rows in one kernel.  Every block makes the
// choice and the order for itself, so that no block waits for another; the first one leaves them for the kernels behind, and
// each copies its share of the rows.
constexpr int DISPATCH_THREADS = 256, DISPATCH_PAIRS = 256, DISPATCH_TOKENS = 32;

template <typename T>
__global__ void __launch_bounds__(DISPATCH_THREADS)
moe_dispatch_kernel(RouteParams p, int* idx, float* weight, int* offsets, int* row_pair, int* pair_row, const T* h, long long ldh,
                    T* rows, long long ldr, int width, int weight_rows, int vec) {
  extern __shared__ float dispatch_sm[];                 // per warp: scores, choice scores, group marks; then counts [n_out + 1]
  __shared__ int s_idx[DISPATCH_PAIRS], s_row[DISPATCH_PAIRS];
  __shared__ float s_w[DISPATCH_PAIRS];
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = DISPATCH_THREADS / 32;
  const int pairs = p.n * p.top;
  float* s = dispatch_sm + (size_t)warp * (2 * p.n_out + p.groups);
  for (int t = warp; t < p.n; t += warps) route_token(p, t, s, s + p.n_out, s + 2 * p.n_out, lane, s_idx + t * p.top, s_w + t * p.top);
  int* start = reinterpret_cast<int*>(dispatch_sm + (size_t)warps * (2 * p.n_out + p.groups));
  __syncthreads();
  // first row of every output's range, and behind the last one: pairs of outputs in front of it
  for (int e = threadIdx.x; e <= p.n_out; e += DISPATCH_THREADS) {
    int c = 0;
#pragma unroll 8
    for (int q = 0; q < pairs; ++q) c += s_idx[q] < e;
    start[e] = c;
  }
  __syncthreads();
  for (int q = threadIdx.x; q < pairs; q += DISPATCH_THREADS) {
    int r = start[s_idx[q]];
#pragma unroll 8
    for (int o = 0; o < q; ++o) r += s_idx[o] == s_idx[q];
    s_row[q] = r;
  }
  __syncthreads();
  if (blockIdx.x == 0) {
    for (int e = threadIdx.x; e <= p.n_out; e += DISPATCH_THREADS) offsets[e] = start[e];
    for (int q = threadIdx.x; q < pairs; q += DISPATCH_THREADS) {
      idx[q] = s_idx[q];
      weight[q] = s_w[q];
      pair_row[q] = s_row[q];
      row_pair[s_row[q]] = q;
    }
  }
  for (int q = blockIdx.x; q < pairs; q += gridDim.x) {
    const float w = weight_rows ? s_w[q] : 1.f;
    const T* src = h + (size_t)(q / p.top) * ldh;
    T* dst = rows + (size_t)s_row[q] * ldr;
    if (vec && !weight_rows) {
      copy_row16(src, dst, width * (int)sizeof(T) / 16);
      continue;
    }
    for (int d = threadIdx.x; d < width; d += DISPATCH_THREADS) dst[d] = from_f32<T>(w * to_f32(src[d]));
  }
}

// one block
__global__ void moe_sort_kernel(const int* idx, int pairs, int E, int* offsets, int* row_pair, int* pair_row) {
  __shared__ int count[MOE_MAX_EXPERTS + 1];
  pdl_trigger();
  pdl_wait();
  for (int e = threadIdx.x; e <= E; e += blockDim.x) count[e] = 0;
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) atomicAdd(&count[idx[p]], 1);
  __syncthreads();
  if (threadIdx.x == 0) {
    int at = 0;
    for (int e = 0; e < E; ++e) {
      const int c = count[e];
      offsets[e] = at;
      count[e] = at;
      at += c;
    }
    offsets[E] = at;
  }
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
    const int row = atomicAdd(&count[idx[p]], 1);
    row_pair[row] = p;
    pair_row[p] = row;
  }
}

// several rows a block: `lanes` neighbouring threads (whole warps) a row
__global__ void moe_gather16_kernel(const char* h, long long ldh_bytes, const int* row_pair, char* rows, long long ldr_bytes, int pairs,
                                    int pieces, int top, int lanes) {
  pdl_trigger();
  const int row = blockIdx.x * (blockDim.x / lanes) + threadIdx.x / lanes;
  pdl_wait();
  if (row >= pairs) return;
  const uint4* src = reinterpret_cast<const uint4*>(h + (size_t)(row_pair[row] / top) * ldh_bytes);
  uint4* dst = reinterpret_cast<uint4*>(rows + (size_t)row * ldr_bytes);
  for (int i = threadIdx.x % lanes; i < pieces; i += lanes) dst[i] = src[i];
}

template <typename T>
__global__ void moe_gather_kernel(const T* h, long long ldh, const int* row_pair, const float* weight, T* rows,
                                  long long ldr, int pairs, int width, int top) {
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x;
  const int p = row_pair[row];
  const float w = weight ? weight[p] : 1.f;              // (no weights: they multiply the experts' outputs instead)
  const T* src = h + (size_t)(p / top) * ldh;
  T* dst = rows + (size_t)row * ldr;
  for (int d = threadIdx.x; d < width; d += blockDim.x) dst[d] = from_f32<T>(w * to_f32(src[d]));
}

// The block's (expert, first row) among the tiles of all experts' ranges, or false.
__device__ __forceinline__ bool moe_tile(const int* offsets, int E, int tile, int& e, int& r0, int& r1) {
  for (e = 0; e < E; ++e) {
    const int lo = offsets[e], hi = offsets[e + 1];
    const int tiles = (hi - lo + 63) >> 6;
    if (tile < tiles) {
      r0 = lo + 64 * tile;
      r1 = hi;
      return true;
    }
    tile -= tiles;
  }
  return false;
}

// GLU: tile columns alternate gate, up, gate, up, ... of 32 features; out [rows, ff]
template <typename TA, typename TW>
__global__ void moe_experts_glu_kernel(const TA* rows, long long ldr, const TW* __restrict__ W, const int* offsets, int E,
                                       TA* act, long long lda, int ff, int width, float alpha, float limit, float up_add,
                                       int blocks64) {
  pdl_trigger();
  pdl_wait();
  int e, r0, r1;
  if (!moe_tile(offsets, E, blockIdx.y, e, r0, r1)) return;
  const int c0 = blockIdx.x * 32;
  const TW* wb = W + (size_t)e * 2 * ff * width;       // [gate rows (ff) | up rows (ff)]
  float acc[4][4];
  int ty, tx;
  hy_tile_64x64<TA, TW>(
      [&](int i) -> const TA* { return r0 + i < r1 ? rows + (size_t)(r0 + i) * ldr : nullptr; },
      [&](int j) -> const TW* {
        const int c = c0 + (j >> 1);
        // rows [gate (ff) | up (ff)], or alternating in blocks of 64: gate 0-63, up 0-63, gate 64-127, ...
        const size_t wrow = blocks64 ? (size_t)(c >> 6) * 128 + (j & 1) * 64 + (c & 63) : (size_t)(j & 1) * ff + c;
        return c < ff ? wb + wrow * width : nullptr;
      },
      width, acc, ty, tx);
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const int row = r0 + ty * 4 + r;
    if (row >= r1) continue;
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      const int col = c0 + tx * 2 + c;
      if (col < ff)
        act[(size_t)row * lda + col] = from_f32<TA>(hy_clamped_glu(acc[r][2 * c], acc[r][2 * c + 1], alpha, limit, up_add));
    }
  }
}

// out = rows W^T (32-bit), or function(rows W^T) in the rows' type
template <typename TA, typename TW, typename TO>
__global__ void moe_experts_down_kernel(const TA* act, long long lda, const TW* __restrict__ W, const int* offsets, int E,
                                        TO* out, long long ldo, int width, int ff, int fn) {
  pdl_trigger();
  pdl_wait();
  int e, r0, r1;
  if (!moe_tile(offsets, E, blockIdx.y, e, r0, r1)) return;
  const int c0 = blockIdx.x * 64;
  const TW* wb = W + (size_t)e * width * ff;
  float acc[4][4];
  int ty, tx;
  hy_tile_64x64<TA, TW>(
      [&](int i) -> const TA* { return r0 + i < r1 ? act + (size_t)(r0 + i) * lda : nullptr; },
      [&](int j) -> const TW* { return c0 + j < width ? wb + (size_t)(c0 + j) * ff : nullptr; }, ff, acc, ty, tx);
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const int row = r0 + ty * 4 + r;
    if (row >= r1) continue;
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int col = c0 + tx * 4 + c;
      if (col < width) out[(size_t)row * ldo + col] = from_f32<TO>(hy_act(acc[r][c], fn));
    }
  }
}

__global__ void moe_combine_kernel(const float* out, long long ldo, const int* pair_row, const float* shared_gate,
                                   const float* shared, long long lds, float* y, long long ldy, int width, int top) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const float g = shared_gate ? shared_gate[t] : 0.f;
  for (int d = threadIdx.x; d < width; d += blockDim.x) {
    float v = 0.f;
    for (int k = 0; k < top; ++k) v += out[(size_t)pair_row[(size_t)t * top + k] * ldo + d];
    if (shared) v += g * shared[(size_t)t * lds + d];
    y[(size_t)t * ldy + d] = v;
  }
}

// rows of any length; `then`: the norm in front of the next sublayer, of the new row
template <typename T>
__global__ void moe_combine_weighted_any_kernel(const float* out, long long ldo, const int* pair_row, const int* idx,
                                                const float* weight, const T* h, long long ldh, float* y, long long ldy,
                                                int width, int top, int E, int accumulate, const float* shared,
                                                long long lds, int splits, size_t split_stride,
                                                const float* __restrict__ shared_bias, ThenNorm then) {
  __shared__ float scratch[32];
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  float* o = y + t * ldy;
  for (int d = threadIdx.x; d < width; d += blockDim.x) {
    float v = 0.f;
    for (int k = 0; k < top; ++k) {
      const size_t p = t * top + k;
      const float src = idx[p] < E ? out[(size_t)pair_row[p] * ldo + d] : to_f32(h[t * ldh + d]);
      v = fmaf(weight[p], src, v);
    }
    if (splits > 0) {
      float sh;
      const size_t at = t * width + d;
      sum_partials<1>(shared, splits, split_stride, &at, &sh);
      v += shared_bias ? sh + shared_bias[d] : sh;
    } else if (shared) {
      v += shared[t * lds + d];
    }
    o[d] = accumulate ? o[d] + v : v;
  }
  if (then.gain != nullptr) hy_then_norm_row(o, width, then, t, scratch);
}

__device__ __forceinline__ float4 load4_f32(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4_f32(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}

// The same arithmetic per value for rows of 16-byte pieces, the new row in the block's registers.
template <typename T, int NV>
__global__ void __launch_bounds__(256)
moe_combine_weighted_kernel(const float* out, long long ldo, const int* pair_row, const int* idx, const float* weight,
                            const T* h, long long ldh, float* y, long long ldy, int width, int top, int E, int accumulate,
                            const float* shared, long long lds, int splits, size_t split_stride,
                            const float* __restrict__ shared_bias, ThenNorm then) {
  __shared__ float scratch[32];
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  float* o = y + t * ldy;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 v[NV], own[NV], sh[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = 4 * (threadIdx.x + i * blockDim.x);
    v[i] = zero;
    own[i] = d < width && accumulate ? load4_f32(o + d) : zero;
    sh[i] = d < width && shared && splits == 0 ? load4_f32(shared + t * lds + d) : zero;
  }
  for (int u = 0; u < splits; ++u) {                      // (shared: partial tiles [splits][tokens * width])
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = 4 * (threadIdx.x + i * blockDim.x);
      if (d >= width) continue;
      const float4 x = load4_f32(shared + u * split_stride + t * width + d);
      sh[i].x += x.x; sh[i].y += x.y; sh[i].z += x.z; sh[i].w += x.w;
    }
  }
  if (splits > 0 && shared_bias) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = 4 * (threadIdx.x + i * blockDim.x);
      if (d >= width) continue;
      const float4 x = load4_f32(shared_bias + d);
      sh[i].x += x.x; sh[i].y += x.y; sh[i].z += x.z; sh[i].w += x.w;
    }
  }
  // four choices at a time, so that their rows are on their way together
  for (int k0 = 0; k0 < top; k0 += 4) {
    float w[4];
    int row[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const size_t p = t * top + min(k0 + u, top - 1);
      w[u] = k0 + u < top ? weight[p] : 0.f;
      row[u] = idx[p] < E ? pair_row[p] : -1;
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = 4 * (threadIdx.x + i * blockDim.x);
      if (d >= width) continue;
      float4 x[4];
#pragma unroll
      for (int u = 0; u < 4; ++u)
        if (k0 + u < top) x[u] = row[u] >= 0 ? load4_f32(out + (size_t)row[u] * ldo + d) : load4_f32(h + t * ldh + d);
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        if (k0 + u >= top) continue;
        v[i].x = fmaf(w[u], x[u].x, v[i].x); v[i].y = fmaf(w[u], x[u].y, v[i].y);
        v[i].z = fmaf(w[u], x[u].z, v[i].z); v[i].w = fmaf(w[u], x[u].w, v[i].w);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = 4 * (threadIdx.x + i * blockDim.x);
    if (d >= width) continue;
    if (shared) { v[i].x += sh[i].x; v[i].y += sh[i].y; v[i].z += sh[i].z; v[i].w += sh[i].w; }
    if (accumulate) { v[i].x += own[i].x; v[i].y += own[i].y; v[i].z += own[i].z; v[i].w += own[i].w; }
    *reinterpret_cast<float4*>(o + d) = v[i];
  }
  if (then.gain != nullptr) hy_then_norm<NV>(v, width, then, t, scratch);
}

}  // namespace

namespace {

// The router's operands: a0 logits (f32), a1 their row stride, a2 tokens, a3 router outputs (experts and identity outputs), a4
// top, a5 scores (0 sigmoid, 1 softmax, 2 the logits), a6 correction [outputs] (f32) or 0, a7 groups (1: none), a8 groups kept,
// a9 chosen outputs [tokens, top] (int32), a10 their weights (f32), a11 how the chosen scores become weights: 0 as they are, 1
// divided by their sum, 2 their softmax, a12 a group's mark: 0 its largest choice score, 1 the sum of its two largest; f0 factor
// on the weights (0 means 1).  A record with GB_OP_TAKES_PARTIALS: the logits are partial tiles of the product in front.
int route_params(const GbPlanCtx* ctx, const long long* a, const double* f, RouteParams& p) {
  p.logits = op_ptr<const float>(a[0]); p.ld = a[1];
  p.part = ctx->part_splits > 0 ? ctx->part : nullptr;
  p.splits = ctx->part_splits; p.part_bias = ctx->part_bias;
  p.n = (int)a[2]; p.n_out = (int)a[3]; p.top = (int)a[4]; p.scores = (int)a[5];
  p.part_stride = (long long)p.n * p.n_out;
  p.correction = op_ptr<const float>(a[6]);
  p.groups = (int)a[7]; p.keep = (int)a[8];
  p.normalise = (int)a[11]; p.mark_two = (int)a[12];
  p.weight_scale = f[0] != 0.0 ? (float)f[0] : 1.f;
  if (p.groups < 1) p.groups = 1;
  if (p.keep < 1 || p.keep > p.groups) p.keep = p.groups;
  if (p.n_out > MOE_MAX_EXPERTS) GB_FAIL(GB_ERR_ARG, "moe_route_grouped: %d router outputs (at most %d)", p.n_out, MOE_MAX_EXPERTS);
  if (p.n_out % p.groups) GB_FAIL(GB_ERR_ARG, "moe_route_grouped: %d router outputs in %d groups", p.n_out, p.groups);
  if (p.top < 1 || p.top > (p.n_out / p.groups) * p.keep)
    GB_FAIL(GB_ERR_ARG, "moe_route_grouped: top %d of the %d outputs in %d open groups", p.top, (p.n_out / p.groups) * p.keep, p.keep);
  return GB_OK;
}

}  // namespace

// (operands: route_params)
GB_OP(gb_op_moe_route_grouped) {
  RouteParams p;
  if (a[2] <= 0) return 0;
  const int rc = route_params(ctx, a, f, p);
  if (rc < 0) return rc;
  const int warps = 4;
  const size_t smem = sizeof(float) * warps * (2 * (size_t)p.n_out + p.groups);
  gb_launch(moe_route_grouped_kernel, dim3(gb_div_up(p.n, warps)), dim3(32 * warps), smem, ctx->stream, p, op_ptr<int>(a[9]),
            op_ptr<float>(a[10]));
  GB_CHECK_LAUNCH("moe_route_grouped");
  return 1;
}

GB_OP(gb_op_moe_sort);
GB_OP(gb_op_moe_gather);

// The choice, the experts' order and the gathered rows: moe_route_grouped, moe_sort and moe_gather, in one kernel for a step
// of few tokens.  a0 to a12 and f0 as of route_params, a13 offsets [outputs + 1], a14 row -> pair, a15 pair -> row, a16 h, a17 its
// row stride, a18 dtype (of h and rows), a19 rows out, a20 their stride, a21 width; flags bit 0: a row is multiplied by its weight
GB_OP(gb_op_moe_dispatch) {
  RouteParams p;
  if (a[2] <= 0) return 0;
  const int rc = route_params(ctx, a, f, p);
  if (rc < 0) return rc;
  const size_t smem = sizeof(float) * (DISPATCH_THREADS / 32 * (2 * (size_t)p.n_out + p.groups) + p.n_out + 1);
  if (p.n <= DISPATCH_TOKENS && (long long)p.n * p.top <= DISPATCH_PAIRS && smem <= 40 * 1024) {
    const int pairs = p.n * p.top;
    const dim3 grid(pairs < 64 ? pairs : 64);
#define DISPATCH(T)                                                                                                     \
    gb_launch(moe_dispatch_kernel<T>, grid, dim3(DISPATCH_THREADS), smem, ctx->stream, p, op_ptr<int>(a[9]), op_ptr<float>(a[10]), \
              op_ptr<int>(a[13]), op_ptr<int>(a[14]), op_ptr<int>(a[15]), op_ptr<const T>(a[16]), a[17], op_ptr<T>(a[19]), a[20],   \
              (int)a[21], flags & 1, vec)
    const long long size = a[18] == GB_BF16 ? 2 : 4;
    const int vec = ((a[16] | a[19] | a[17] * size | a[20] * size | a[21] * size) & 15) == 0;
    if (a[18] == GB_BF16) DISPATCH(bf16); else DISPATCH(float);
#undef DISPATCH
    GB_CHECK_LAUNCH("moe_dispatch");
    return 1;
  }
  const int r1 = gb_op_moe_route_grouped(ctx, a, f, 0);
  if (r1 < 0) return r1;
  const long long so[24] = {a[9], a[2], a[3], a[13], a[14], a[15], a[4]};
  const int r2 = gb_op_moe_sort(ctx, so, f, 0);
  if (r2 < 0) return r2;
  const long long ga[24] = {a[16], a[17], a[18], a[14], (flags & 1) ? a[10] : 0, a[19], a[20], a[2], a[21], a[4]};
  const int r3 = gb_op_moe_gather(ctx, ga, f, 0);
  return r3 < 0 ? r3 : r1 + r2 + r3;
}

// a0 logits (f32), a1 their row stride, a2 tokens, a3 experts, a4 top, a5 column of the shared expert's gate logit,
// a6 chosen experts [tokens, top] (int32), a7 their weights (f32), a8 shared gate [tokens] (f32), or 0 for none
GB_OP(gb_op_moe_route) {
  const int n = (int)a[2], E = (int)a[3], top = (int)a[4];
  if (n <= 0) return 0;
  if (top < 1 || top > E) GB_FAIL(GB_ERR_ARG, "moe_route: top %d of %d experts", top, E);
  if (E > MOE_MAX_EXPERTS) GB_FAIL(GB_ERR_ARG, "moe_route: %d experts (at most %d)", E, MOE_MAX_EXPERTS);
  gb_launch(moe_route_kernel, dim3(gb_div_up(n, 4)), dim3(128), 0, ctx->stream, op_ptr<const float>(a[0]), a[1], n, E,
            top, (int)a[5], op_ptr<int>(a[6]), op_ptr<float>(a[7]), op_ptr<float>(a[8]));
  GB_CHECK_LAUNCH("moe_route");
  return 1;
}

// a0 chosen experts [tokens, top], a1 tokens, a2 experts, a3 offsets [E + 1], a4 row -> pair, a5 pair -> row, a6 top
GB_OP(gb_op_moe_sort) {
  const int pairs = (int)(a[1] * a[6]), E = (int)a[2];
  if (pairs <= 0) return 0;
  if (E > MOE_MAX_EXPERTS) GB_FAIL(GB_ERR_ARG, "moe_sort: %d experts (at most %d)", E, MOE_MAX_EXPERTS);
  gb_launch(moe_sort_kernel, dim3(1), dim3(1024), 0, ctx->stream, op_ptr<const int>(a[0]), pairs, E, op_ptr<int>(a[3]),
            op_ptr<int>(a[4]), op_ptr<int>(a[5]));
  GB_CHECK_LAUNCH("moe_sort");
  return 1;
}

// a0 h, a1 its row stride, a2 dtype (of h and rows), a3 row -> pair, a4 weights [pairs] or 0 (plain copies), a5 rows out, a6 their
// stride, a7 tokens, a8 width, a9 top
GB_OP(gb_op_moe_gather) {
  const int pairs = (int)(a[7] * a[9]), width = (int)a[8];
  if (pairs <= 0) return 0;
  const dim3 grid(pairs), block(width <= 256 ? 64 : 256);
  const long long size = a[2] == GB_BF16 ? 2 : 4;
  if (!a[4] && ((a[0] | a[5] | a[1] * size | a[6] * size | width * size) & 15) == 0) {
    const int pieces = (int)(width * size / 16), lanes = pieces >= 128 ? 128 : pieces >= 64 ? 64 : 32;
    gb_launch(moe_gather16_kernel, dim3(gb_div_up(pairs, 256 / lanes)), dim3(256), 0, ctx->stream, op_ptr<const char>(a[0]), a[1] * size,
              op_ptr<const int>(a[3]), op_ptr<char>(a[5]), a[6] * size, pairs, pieces, (int)a[9], lanes);
    GB_CHECK_LAUNCH("moe_gather");
    return 1;
  }
  if (a[2] == GB_BF16)
    gb_launch(moe_gather_kernel<bf16>, grid, block, 0, ctx->stream, op_ptr<const bf16>(a[0]), a[1], op_ptr<const int>(a[3]),
              op_ptr<const float>(a[4]), op_ptr<bf16>(a[5]), a[6], pairs, width, (int)a[9]);
  else
    gb_launch(moe_gather_kernel<float>, grid, block, 0, ctx->stream, op_ptr<const float>(a[0]), a[1], op_ptr<const int>(a[3]),
              op_ptr<const float>(a[4]), op_ptr<float>(a[5]), a[6], pairs, width, (int)a[9]);
  GB_CHECK_LAUNCH("moe_gather");
  return 1;
}

// a0 input rows, a1 their stride, a2 their dtype, a3 weights [E, out features, in features], a4 their dtype,
// a5 offsets [E + 1], a6 experts, a7 out, a8 its row stride, a9 tokens, a10 features out (GLU: ff), a11 features in,
// a12 mode (0: GLU over [gate rows | up rows], out in the input's dtype; 1: plain, out f32; 2: a function of the sums, out
// in the input's dtype), a13 top, a14 (GLU) 1 when gate and up rows alternate in blocks of 64 instead, (mode 2) the
// function's number; f0 alpha, f1 limit, f2 what is added to u
GB_OP(gb_op_moe_experts) {
  const int pairs = (int)(a[9] * a[13]), E = (int)a[6], n_out = (int)a[10], n_in = (int)a[11], mode = (int)a[12];
  if (pairs <= 0) return 0;
  const int tiles = gb_div_up(pairs, 64) + E;            // at most this many row tiles over all experts
  const bool abf = a[2] == GB_BF16, wbf = a[4] == GB_BF16;
  if (abf && !wbf) GB_FAIL(GB_ERR_ARG, "moe_experts: bfloat16 rows with 32-bit weights");
#define GLU(TA, TW)                                                                                                 \
  gb_launch(moe_experts_glu_kernel<TA, TW>, dim3(gb_div_up(n_out, 32), tiles), dim3(256), 0, ctx->stream,          \
            op_ptr<const TA>(a[0]), a[1], op_ptr<const TW>(a[3]), op_ptr<const int>(a[5]), E, op_ptr<TA>(a[7]), a[8], \
            n_out, n_in, (float)f[0], (float)f[1], (float)f[2], (int)a[14])
#define DOWN(TA, TW, TO, FN)                                                                                        \
  gb_launch(moe_experts_down_kernel<TA, TW, TO>, dim3(gb_div_up(n_out, 64), tiles), dim3(256), 0, ctx->stream,     \
            op_ptr<const TA>(a[0]), a[1], op_ptr<const TW>(a[3]), op_ptr<const int>(a[5]), E, op_ptr<TO>(a[7]),      \
            a[8], n_out, n_in, FN)
  if (mode == 0) {
    if (abf) GLU(bf16, bf16); else if (wbf) GLU(float, bf16); else GLU(float, float);
  } else if (mode == 2) {
    const int fn = (int)a[14];
    if (fn < 0 || fn > ACT_NONE) GB_FAIL(GB_ERR_ARG, "moe_experts: function %d", fn);
    if (abf) DOWN(bf16, bf16, bf16, fn); else if (wbf) DOWN(float, bf16, float, fn); else DOWN(float, float, float, fn);
  } else {
    if (abf) DOWN(bf16, bf16, float, ACT_NONE); else if (wbf) DOWN(float, bf16, float, ACT_NONE);
    else DOWN(float, float, float, ACT_NONE);
  }
#undef GLU
#undef DOWN
  GB_CHECK_LAUNCH("moe_experts");
  return 1;
}

// a0 expert outputs by row (f32), a1 their stride, a2 pair -> row, a3 shared gate [tokens] or 0, a4 shared expert's
// output (f32) or 0, a5 its row stride, a6 y (f32), a7 its row stride, a8 tokens, a9 width, a10 top
GB_OP(gb_op_moe_combine) {
  const int n = (int)a[8], width = (int)a[9];
  if (n <= 0) return 0;
  gb_launch(moe_combine_kernel, dim3(n), dim3(width <= 256 ? 64 : 256), 0, ctx->stream, op_ptr<const float>(a[0]), a[1],
            op_ptr<const int>(a[2]), op_ptr<const float>(a[3]), op_ptr<const float>(a[4]), a[5], op_ptr<float>(a[6]), a[7],
            width, (int)a[10]);
  GB_CHECK_LAUNCH("moe_combine");
  return 1;
}

// a0 expert outputs by row (f32), a1 their stride, a2 pair -> row, a3 chosen outputs [tokens, top], a4 their weights,
// a5 the feed-forward's input h, a6 its row stride, a7 its dtype, a8 y (f32), a9 its row stride, a10 tokens, a11 width,
// a12 top, a13 real experts (a choice from here on returns h), a14 an output added for every token (f32) or 0, a15 its row
// stride, a16 gain of a norm taken of the new rows or 0: none, a17 its output [tokens, width], a18 that dtype, a19 its kind
// (0 layer norm, 1 RMS norm), a20 its eps (the bits of a 32-bit float); flags bit 0: add into y.  A record with
// GB_OP_TAKES_PARTIALS: a14's output may be partial tiles of the product in front
GB_OP(gb_op_moe_combine_weighted) {
  const int n = (int)a[10], width = (int)a[11];
  if (n <= 0) return 0;
  const ThenNorm then = hy_then_of(a[16], a[17], a[18], a[19], a[20]);
  const int splits = a[14] ? ctx->part_splits : 0;
  const float* shared = splits > 0 ? ctx->part : op_ptr<const float>(a[14]);
  const float* shared_bias = splits > 0 ? ctx->part_bias : nullptr;
  const size_t split_stride = (size_t)n * width;
  const bool vec = (((uintptr_t)shared | (uintptr_t)shared_bias) & 15) == 0 && width % 4 == 0 && width <= 4096 && a[1] % 4 == 0 && a[6] % 4 == 0 && a[9] % 4 == 0 && a[15] % 4 == 0 &&
                   ((a[0] | a[8] | a[14]) & 15) == 0 && (a[5] & (a[7] == GB_BF16 ? 7 : 15)) == 0 && hy_then_vec(then);
#define COMBINE(T, KERNEL, THREADS)                                                                                     \
  gb_launch(KERNEL, dim3(n), dim3(THREADS), 0, ctx->stream, op_ptr<const float>(a[0]), a[1], op_ptr<const int>(a[2]),    \
            op_ptr<const int>(a[3]), op_ptr<const float>(a[4]), op_ptr<const T>(a[5]), a[6], op_ptr<float>(a[8]), a[9],  \
            width, (int)a[12], (int)a[13], flags & 1, shared, a[15], splits, split_stride, shared_bias, then)
  const int threads = hy_row_threads(width);
#define COMBINE_OF(T)                                                                                                   \
  do {                                                                                                                  \
    if (!vec) COMBINE(T, moe_combine_weighted_any_kernel<T>, width <= 256 ? 64 : 256);                                  \
    else if (width <= 4 * threads) COMBINE(T, (moe_combine_weighted_kernel<T, 1>), threads);                            \
    else if (width <= 8 * threads) COMBINE(T, (moe_combine_weighted_kernel<T, 2>), threads);                            \
    else COMBINE(T, (moe_combine_weighted_kernel<T, 4>), threads);                                                      \
  } while (0)
  if (a[7] == GB_BF16) COMBINE_OF(bf16); else COMBINE_OF(float);
#undef COMBINE_OF
#undef COMBINE
  GB_CHECK_LAUNCH("moe_combine_weighted");
  return 1;
}
