// Residual streams that are mixed by small matrices (hyper-connections): instead of one residual row of `dim` values a
// token has `streams` of them, side by side in one row of the 32-bit stream.
//
//  gb_op_stream_read   what a sublayer reads: u = sum_s in[s] * x_s, then h = rmsnorm(u) * gain.  Without `in` the
//                      weights are ones (the sum of the streams, in front of the head); the rows may be gathered.
//  gb_op_stream_mix    what a sublayer leaves: x_t <- sum_s mix[s][t] * x_s + out[t] * y, all streams from the old
//                      ones, and, while the new rows are in registers, what the NEXT sublayer reads of them
//                      (its own u and norm), so that a row of streams is read and written once a sublayer.
//
// A thread walks pieces of VEC neighbouring values (four where rows allow, else one) and handles all streams of a
// piece itself, so the in-place update needs no exchange between threads; the norm needs one block-wide sum.
#include "hybrid.cuh"

namespace {

constexpr int MAX_STREAMS = 16;

template <int VEC> struct Piece;
template <> struct Piece<1> {
  float v[1];
  __device__ __forceinline__ void load(const float* p) { v[0] = *p; }
  __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
};
template <> struct Piece<4> {
  float v[4];
  __device__ __forceinline__ void load(const float* p) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
  }
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};

template <int VEC>
__device__ __forceinline__ void store_normed(void* out, int dtype, size_t at, const float* u, float rstd, const float* gain) {
  if (dtype == GB_BF16) {
    bf16* o = (bf16*)out + at;
    if constexpr (VEC == 4) {
      __nv_bfloat162 lo = __floats2bfloat162_rn(u[0] * rstd * gain[0], u[1] * rstd * gain[1]);
      __nv_bfloat162 hi = __floats2bfloat162_rn(u[2] * rstd * gain[2], u[3] * rstd * gain[3]);
      uint2 w;
      w.x = *reinterpret_cast<unsigned*>(&lo);
      w.y = *reinterpret_cast<unsigned*>(&hi);
      *reinterpret_cast<uint2*>(o) = w;
    } else {
      *o = __float2bfloat16_rn(u[0] * rstd * gain[0]);
    }
  } else {
    float* o = (float*)out + at;
#pragma unroll
    for (int e = 0; e < VEC; ++e) o[e] = u[e] * rstd * gain[e];
  }
}

struct StreamParams {
  float* x; long long ldx;                 // [rows, streams * dim]
  const float* y; long long ldy;           // a sublayer's output (mixing only)
  const float* part; int splits;           // or its partial tiles [splits][rows][dim], added up in this order
  long long part_stride; const float* part_bias;
  const float* mix;                        // [streams][streams], from x to
  const float* out_w;                      // [streams]
  const float* in_w;                       // [streams] weights of the next reader, or null: ones
  const float* gain;                       // its norm's gain, or null: nothing is read
  void* out; int out_dtype;
  const int* rows;                         // row list (reading only) or null
  int dim; float eps;
};

constexpr int STREAM_CACHE = 4;            // pieces of u a thread keeps between the sum of squares and the norm

// S streams (0: any number up to MAX_STREAMS, taken from `streams`); PART: y comes as partial tiles.
template <int S, int VEC, bool MIX, bool PART>
__global__ void stream_kernel(StreamParams p, int streams) {
  constexpr int CAP = S > 0 ? S : MAX_STREAMS;
  __shared__ float scratch[32];
  __shared__ float w_mix[MIX ? CAP * CAP : 1], w_out[MIX ? CAP : 1], w_in[CAP];
  pdl_trigger();
  const int n_s = S > 0 ? S : streams;
  // (weights: nothing writes them while a model runs)
  for (int i = threadIdx.x; i < n_s; i += blockDim.x) {
    w_in[i] = p.in_w ? p.in_w[i] : 1.f;
    if (MIX) w_out[i] = p.out_w[i];
  }
  if (MIX)
    for (int i = threadIdx.x; i < n_s * n_s; i += blockDim.x) w_mix[i] = p.mix[i];
  const int r = blockIdx.x;
  const int src = p.rows ? p.rows[r] : r;
  __syncthreads();
  float m[S > 0 && S <= 4 ? S * S : 1], wo[S > 0 && S <= 4 ? S : 1], wi[S > 0 && S <= 4 ? S : 1];
  if constexpr (S > 0 && S <= 4) {                       // few streams: the weights live in registers
#pragma unroll
    for (int i = 0; i < S; ++i) {
      wi[i] = w_in[i];
      if (MIX) wo[i] = w_out[i];
    }
    if (MIX) {
#pragma unroll
      for (int i = 0; i < S * S; ++i) m[i] = w_mix[i];
    }
  }
  pdl_wait();
  float* x = p.x + (size_t)src * p.ldx;
  const float* y = MIX ? p.y + (size_t)r * p.ldy : nullptr;
  const int pieces = p.dim / VEC;
  float cache[STREAM_CACHE][VEC];
  float ss = 0.f;
  auto read = [&](const Piece<VEC>* v, float* u) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) u[e] = 0.f;
#pragma unroll
    for (int s = 0; s < CAP; ++s) {
      if (S == 0 && s >= n_s) break;
      float w;
      if constexpr (S > 0 && S <= 4) w = wi[s]; else w = w_in[s];
#pragma unroll
      for (int e = 0; e < VEC; ++e) u[e] = fmaf(w, v[s].v[e], u[e]);
    }
  };
  auto step = [&](int i, float* u) {                     // piece i: mixed and stored, then read
    Piece<VEC> old[CAP];
#pragma unroll
    for (int s = 0; s < CAP; ++s)
      if (S > 0 || s < n_s) old[s].load(x + (size_t)s * p.dim + (size_t)i * VEC);
    if constexpr (MIX) {
      Piece<VEC> yy, now[CAP];
      if constexpr (!PART) {
        yy.load(y + (size_t)i * VEC);
      } else {
        const float* at = p.part + (size_t)r * p.dim + (size_t)i * VEC;
#pragma unroll
        for (int e = 0; e < VEC; ++e) yy.v[e] = 0.f;
        for (int s0 = 0; s0 < p.splits; s0 += 4) {         // (four requested together, added in order)
          Piece<VEC> t[4];
#pragma unroll
          for (int u = 0; u < 4; ++u) t[u].load(at + (size_t)min(s0 + u, p.splits - 1) * p.part_stride);
#pragma unroll
          for (int u = 0; u < 4; ++u)
            if (s0 + u < p.splits) {
#pragma unroll
              for (int e = 0; e < VEC; ++e) yy.v[e] += t[u].v[e];
            }
        }
        if (p.part_bias) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) yy.v[e] += p.part_bias[(size_t)i * VEC + e];
        }
      }
#pragma unroll
      for (int t = 0; t < CAP; ++t) {
        if (S == 0 && t >= n_s) break;
        float a[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) a[e] = 0.f;
#pragma unroll
        for (int s = 0; s < CAP; ++s) {
          if (S == 0 && s >= n_s) break;
          float w;
          if constexpr (S > 0 && S <= 4) w = m[s * S + t]; else w = w_mix[s * n_s + t];
#pragma unroll
          for (int e = 0; e < VEC; ++e) a[e] = fmaf(w, old[s].v[e], a[e]);
        }
        float w;
        if constexpr (S > 0 && S <= 4) w = wo[t]; else w = w_out[t];
#pragma unroll
        for (int e = 0; e < VEC; ++e) now[t].v[e] = fmaf(w, yy.v[e], a[e]);
        now[t].store(x + (size_t)t * p.dim + (size_t)i * VEC);
      }
      if (p.gain) read(now, u);
    } else {
      read(old, u);
    }
  };
#pragma unroll
  for (int c = 0; c < STREAM_CACHE; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
#pragma unroll
    for (int e = 0; e < VEC; ++e) cache[c][e] = 0.f;
    if (i < pieces) step(i, cache[c]);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(cache[c][e], cache[c][e], ss);
  }
  for (int i = threadIdx.x + STREAM_CACHE * blockDim.x; i < pieces; i += blockDim.x) {
    float u[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) u[e] = 0.f;
    step(i, u);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(u[e], u[e], ss);
  }
  if (p.gain == nullptr) return;
  const float rstd = 1.0f / sqrtf(block_sum(ss, scratch) / (float)p.dim + p.eps);
#pragma unroll
  for (int c = 0; c < STREAM_CACHE; ++c) {
    const int i = threadIdx.x + c * blockDim.x;
    if (i >= pieces) continue;
    Piece<VEC> g;
    g.load(p.gain + (size_t)i * VEC);
    store_normed<VEC>(p.out, p.out_dtype, (size_t)r * p.dim + (size_t)i * VEC, cache[c], rstd, g.v);
  }
  // (a row too long for the registers: what this thread wrote is read again)
  for (int i = threadIdx.x + STREAM_CACHE * blockDim.x; i < pieces; i += blockDim.x) {
    Piece<VEC> v[CAP], g;
    float u[VEC];
#pragma unroll
    for (int s = 0; s < CAP; ++s)
      if (S > 0 || s < n_s) v[s].load(x + (size_t)s * p.dim + (size_t)i * VEC);
    read(v, u);
    g.load(p.gain + (size_t)i * VEC);
    store_normed<VEC>(p.out, p.out_dtype, (size_t)r * p.dim + (size_t)i * VEC, u, rstd, g.v);
  }
}

template <bool MIX>
int launch_streams(const StreamParams& p, int n, int streams, cudaStream_t stream, const char* what) {
  if (streams < 1 || streams > MAX_STREAMS) GB_FAIL(GB_ERR_ARG, "%s: %d streams (1 to %d)", what, streams, MAX_STREAMS);
  const uintptr_t bits = (uintptr_t)p.x | (uintptr_t)p.y | (uintptr_t)p.gain | (uintptr_t)p.part;
  const bool vec = p.dim % 4 == 0 && p.ldx % 4 == 0 && p.ldy % 4 == 0 && (bits & 15) == 0 &&
                   ((uintptr_t)p.out & (p.out_dtype == GB_BF16 ? 7 : 15)) == 0;
  const int pieces = vec ? p.dim / 4 : p.dim;
  const dim3 block(pieces <= 64 ? 64 : pieces <= 256 ? 128 : 256);
#define STREAMS(S)                                                                                       \
  do {                                                                                                   \
    if (MIX && p.part) {                                                                                 \
      if (vec) gb_launch(stream_kernel<S, 4, MIX, MIX>, dim3(n), block, 0, stream, p, streams);          \
      else gb_launch(stream_kernel<S, 1, MIX, MIX>, dim3(n), block, 0, stream, p, streams);              \
    } else {                                                                                             \
      if (vec) gb_launch(stream_kernel<S, 4, MIX, false>, dim3(n), block, 0, stream, p, streams);        \
      else gb_launch(stream_kernel<S, 1, MIX, false>, dim3(n), block, 0, stream, p, streams);            \
    }                                                                                                    \
  } while (0)
  switch (streams) {
    case 1: STREAMS(1); break;
    case 2: STREAMS(2); break;
    case 3: STREAMS(3); break;
    case 4: STREAMS(4); break;
    case 8: STREAMS(8); break;
    default: STREAMS(0);
  }
#undef STREAMS
  GB_CHECK_LAUNCH(what);
  return 1;
}

}  // namespace

// a0 x (f32 [rows, streams * dim]), a1 its row stride, a2 weights of the streams [streams] (f32) or 0: ones, a3 gain
// [dim], a4 out [rows, dim], a5 out dtype, a6 row list (int32) or 0, a7 rows, a8 dim, a9 streams; f0 eps
GB_OP(gb_op_stream_read) {
  if (a[7] <= 0) return 0;
  StreamParams p{};
  p.x = op_ptr<float>(a[0]); p.ldx = a[1]; p.in_w = op_ptr<const float>(a[2]); p.gain = op_ptr<const float>(a[3]);
  p.out = op_ptr<void>(a[4]); p.out_dtype = (int)a[5]; p.rows = op_ptr<const int>(a[6]);
  p.dim = (int)a[8]; p.eps = (float)f[0];
  return launch_streams<false>(p, (int)a[7], (int)a[9], ctx->stream, "stream_read");
}

// a0 x (f32 [rows, streams * dim], changed in place), a1 its row stride, a2 y (f32 [rows, dim]), a3 its row stride,
// a4 mix [streams][streams] (f32: from the first index to the second), a5 weights of y [streams], a6 rows, a7 dim,
// a8 streams; what the next sublayer reads of the new streams: a9 its weights [streams] or 0: ones, a10 its norm's gain
// or 0: nothing is read, a11 out [rows, dim], a12 out dtype; f0 that norm's eps.  A record with GB_OP_TAKES_PARTIALS: y
// may be the partial tiles of the product in front
GB_OP(gb_op_stream_mix) {
  if (a[6] <= 0) return 0;
  StreamParams p{};
  p.x = op_ptr<float>(a[0]); p.ldx = a[1]; p.y = op_ptr<const float>(a[2]); p.ldy = a[3];
  if (ctx->part_splits > 0) {
    p.part = ctx->part; p.splits = ctx->part_splits;
    p.part_stride = a[6] * a[7]; p.part_bias = ctx->part_bias;
  }
  p.mix = op_ptr<const float>(a[4]); p.out_w = op_ptr<const float>(a[5]);
  p.dim = (int)a[7]; p.in_w = op_ptr<const float>(a[9]); p.gain = op_ptr<const float>(a[10]);
  p.out = op_ptr<void>(a[11]); p.out_dtype = (int)a[12]; p.eps = (float)f[0];
  return launch_streams<true>(p, (int)a[6], (int)a[8], ctx->stream, "stream_mix");
}
