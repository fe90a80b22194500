// Shared pieces of the "hybrid" kernel library: layer norms, gated linear units with clamps, latent
// attention, state-space recurrences and routed experts.
//
// Every exported operation has the signature of a step-plan operation (gb_plan_op.h):
//
//     int gb_op_xxx(const GbPlanCtx* ctx, const long long* a, const double* f, int flags)
//
// so that ONE entry point serves both ways of running a model: the step walker calls it with a
// record's operands (symbols already replaced by the step's values), and the Python wrappers call it
// directly with the same operand list.  It launches on ctx->stream and returns the number of kernels
// launched, or a negative code with the message in gb_last_error().
#pragma once
#include <cstring>

#include "common.cuh"
#include "gb_plan_op.h"

#define GB_OP(name) GB_API int name(const GbPlanCtx* ctx, const long long* a, const double* f, int flags)

template <typename T> static inline T* op_ptr(long long v) { return reinterpret_cast<T*>(v); }

__device__ __forceinline__ float hy_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float hy_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float hy_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float hy_gelu(float z) { return 0.5f * z * (1.0f + erff(z * 0.7071067811865476f)); }
__device__ __forceinline__ float hy_gelu_tanh(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// g' = min(g, limit), u' = clamp(u, -limit, limit): g' * sigmoid(alpha * g') * (u' + up_add)
__device__ __forceinline__ float hy_clamped_glu(float g, float u, float alpha, float limit, float up_add) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * hy_sigmoid(alpha * g) * (u + up_add);
}

// Functions of a feed-forward's units by number.
enum { ACT_GELU_ERF = 0, ACT_GELU_TANH = 1, ACT_SILU = 2, ACT_RELU = 3, ACT_RELU2 = 4, ACT_NONE = 5 };

__device__ __forceinline__ float hy_act(float z, int kind) {
  switch (kind) {
    case ACT_GELU_ERF: return hy_gelu(z);
    case ACT_GELU_TANH: return hy_gelu_tanh(z);
    case ACT_SILU: return hy_silu(z);
    case ACT_RELU: return fmaxf(z, 0.f);
    case ACT_RELU2: z = fmaxf(z, 0.f); return z * z;
    default: return z;
  }
}

enum { NORM_LAYER = 0, NORM_RMS = 1 };

// `then`: the norm in front of the NEXT sublayer, taken of the new rows while they are in registers
// (out = norm(x) * gain), so that it needs no kernel and no second trip of its own.
struct ThenNorm {
  const float* gain;
  void* out;
  int out_dtype, kind;
  float eps;
};

// (as five operands of an operation, the last one the bits of the 32-bit eps)
static inline ThenNorm hy_then_of(long long gain, long long out, long long dtype, long long kind, long long eps_bits) {
  ThenNorm t;
  t.gain = op_ptr<const float>(gain);
  t.out = op_ptr<void>(out);
  t.out_dtype = (int)dtype;
  t.kind = (int)kind;
  const unsigned b = (unsigned)eps_bits;
  memcpy(&t.eps, &b, sizeof(float));
  return t;
}
static inline bool hy_then_vec(const ThenNorm& t) {
  return t.gain == nullptr || (((uintptr_t)t.gain | (uintptr_t)t.out) & 15) == 0;
}
// Threads of a block that holds a row of `dim` values in pieces of four (up to 256, whole warps).
static inline int hy_row_threads(int dim) {
  const int t = (dim / 4 + 31) / 32 * 32;
  return t < 32 ? 32 : t > 256 ? 256 : t;
}

// A row in the block's registers, NV pieces of four values a thread (piece i at 4 * (threadIdx.x + i * blockDim.x)).
template <int NV>
__device__ __forceinline__ void hy_then_norm(const float4 (&v)[NV], int dim, const ThenNorm& then, size_t row, float* scratch) {
  float mean = 0.f;
  if (then.kind == NORM_LAYER) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (4 * (int)(threadIdx.x + i * blockDim.x) < dim) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    mean = block_sum(s, scratch) / (float)dim;
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    if (4 * (int)(threadIdx.x + i * blockDim.x) >= dim) continue;
    const float p = v[i].x - mean, q = v[i].y - mean, c = v[i].z - mean, e = v[i].w - mean;
    ss += (p * p + q * q) + (c * c + e * e);
  }
  const float rstd = 1.0f / sqrtf(block_sum(ss, scratch) / (float)dim + then.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = 4 * (threadIdx.x + i * blockDim.x);
    if (d >= dim) continue;
    const float4 g = *reinterpret_cast<const float4*>(then.gain + d);
    const float r0 = (v[i].x - mean) * rstd * g.x, r1 = (v[i].y - mean) * rstd * g.y;
    const float r2 = (v[i].z - mean) * rstd * g.z, r3 = (v[i].w - mean) * rstd * g.w;
    if (then.out_dtype == GB_BF16) {
      __nv_bfloat162 lo = __floats2bfloat162_rn(r0, r1), hi = __floats2bfloat162_rn(r2, r3);
      uint2 w;
      w.x = *reinterpret_cast<unsigned*>(&lo);
      w.y = *reinterpret_cast<unsigned*>(&hi);
      *reinterpret_cast<uint2*>((bf16*)then.out + row * dim + d) = w;
    } else {
      *reinterpret_cast<float4*>((float*)then.out + row * dim + d) = make_float4(r0, r1, r2, r3);
    }
  }
}

// The same for a row of any length that this block's threads have just written, each its own entries threadIdx.x + i * blockDim.x.
__device__ __forceinline__ void hy_then_norm_row(const float* o, int dim, const ThenNorm& then, size_t row, float* scratch) {
  float mean = 0.f;
  if (then.kind == NORM_LAYER) {
    float s = 0.f;
    for (int d = threadIdx.x; d < dim; d += blockDim.x) s += o[d];
    mean = block_sum(s, scratch) / (float)dim;
  }
  float ss = 0.f;
  for (int d = threadIdx.x; d < dim; d += blockDim.x) ss += (o[d] - mean) * (o[d] - mean);
  const float rstd = 1.0f / sqrtf(block_sum(ss, scratch) / (float)dim + then.eps);
  for (int d = threadIdx.x; d < dim; d += blockDim.x) {
    const float h = (o[d] - mean) * rstd * then.gain[d];
    if (then.out_dtype == GB_BF16) ((bf16*)then.out)[row * dim + d] = __float2bfloat16_rn(h);
    else ((float*)then.out)[row * dim + d] = h;
  }
}

// A 64 x 64 tile of C = A . B^T on the CUDA cores in 32-bit, for 256 threads.  Row i of the tile is
// A[arow(i)] (null: a row of zeros), column j is B[brow(j)] (null likewise), both of K contiguous
// elements.  Every output is one accumulator walking k upwards, so a row's result does not depend on
// which other rows share its tile.  acc[r][c] belongs to tile row ty*4+r, column tx*4+c.
template <typename TA, typename TB, typename ARow, typename BRow>
__device__ __forceinline__ void hy_tile_64x64(ARow arow, BRow brow, int K, float (&acc)[4][4], int& ty, int& tx) {
  __shared__ float As[32][65];          // [k][row]
  __shared__ float Bs[32][65];          // [k][col]
  const int tid = threadIdx.x;
  ty = tid >> 4;
  tx = tid & 15;
#pragma unroll
  for (int r = 0; r < 4; ++r)
#pragma unroll
    for (int c = 0; c < 4; ++c) acc[r][c] = 0.f;
  // loading: thread (lr, lk) fetches rows lr, lr+8, ... at k offset lk
  const int lk = tid & 31, lr = tid >> 5;
  for (int k0 = 0; k0 < K; k0 += 32) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int row = lr + 8 * i;
      const TA* ap = arow(row);
      const TB* bp = brow(row);
      const int k = k0 + lk;
      As[lk][row] = (ap != nullptr && k < K) ? to_f32(ap[k]) : 0.f;
      Bs[lk][row] = (bp != nullptr && k < K) ? to_f32(bp[k]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int kk = 0; kk < 32; ++kk) {
      float av[4], bv[4];
#pragma unroll
      for (int r = 0; r < 4; ++r) av[r] = As[kk][ty * 4 + r];
#pragma unroll
      for (int c = 0; c < 4; ++c) bv[c] = Bs[kk][tx * 4 + c];
#pragma unroll
      for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[r][c] = fmaf(av[r], bv[c], acc[r][c]);
    }
    __syncthreads();
  }
}
