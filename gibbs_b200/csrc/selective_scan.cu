// A selective scan: a diagonal state-space recurrence per channel with inputs, step sizes and read-outs that depend on
// the token, over a ragged batch of prompt portions and single decoded tokens, with per-request state in slots.
// Per channel c and state entry n (32-bit, zero for a new request), token after token:
//
//     dt      = softplus(dt_raw[c] + dt_bias[c])
//     S[c, n] <- exp(dt A[c, n]) S[c, n] + dt x[c] B[n],     A = -exp(A_log)
//     y[c]    = sum_n S[c, n] C[n] + D[c] x[c],              out[c] = y[c] * silu(z[c])
//
// State layout in a slot: [inner][state].
#include "hybrid.cuh"

namespace {

constexpr int SEL_THREADS = 128, SEL_TOKENS = 16;

struct SelParams {
  const float* x; long long ldx;           // [t, inner], behind the convolution
  const float* dt; long long lddt;         // [t, inner], before bias and softplus
  const float* B; const float* C; long long ldbc;        // [t, state] each
  const float* z; long long ldz;           // [t, inner]
  const float* dt_bias; const float* a_log; const float* dskip;
  float* state; long long slot_stride;
  const int* slot_ids; const int* q_start; const int* q_len;
  void* out; long long ldo;
  int inner, N;
  int vec_bc, vec_x;                       // rows of B and C (of x and dt) can be copied in 16-byte pieces
};

__device__ __forceinline__ void sel_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int LEFT> __device__ __forceinline__ void sel_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(LEFT) : "memory");
}
// e^x for what is kept in bfloat16 around it: the hardware's 2^x (its argument already carries log2 e)
__device__ __forceinline__ float sel_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// SPLIT neighbouring lanes share a channel, PER state entries each (state <= SPLIT * PER; lane q holds entries
// 4 (q + SPLIT i) + e).  B, C, x and the raw step sizes of SEL_TOKENS tokens at a time arrive by asynchronous copies
// into one of two buffers while the tokens of the other are consumed.  Once they have landed the block turns raw step
// sizes into (dt, dt x) in place; the read-outs of a chunk's tokens are left in shared memory, and the block finishes
// them (D x, the gate) with coalesced loads and stores.  The read-outs of GROUP tokens are added over a channel's lanes
// together, every exchange halving what a lane still carries; single tokens at a portion's end are added in the same
// order.  FAST: exponentials of decays as the hardware's 2^x (bfloat16 models); else expf.
template <int SPLIT, int PER, bool FAST, typename TO>
__global__ void __launch_bounds__(SEL_THREADS) selective_scan_kernel(SelParams p) {
  constexpr int NR = SPLIT * PER, CH = SEL_THREADS / SPLIT, Q4 = PER / 4, TOK = SEL_TOKENS;
  constexpr int GROUP = SPLIT < 4 ? SPLIT : 4;
  constexpr int BUF = TOK * (2 * NR + 2 * CH);           // B [TOK][NR] | C [TOK][NR] | x [TOK][CH] | dt [TOK][CH]
  extern __shared__ __align__(16) float sel_sm[];        // [2][BUF], then step sizes [TOK][CH], then read-outs [TOK][CH]
  float* sDt = sel_sm + 2 * BUF;
  float* sY = sDt + TOK * CH;
  pdl_trigger();
  const int ch = threadIdx.x / SPLIT, q = threadIdx.x % SPLIT;
  const int r = blockIdx.x, c0 = blockIdx.y * CH, c = c0 + ch;
  const bool active = c < p.inner;
  const int first = p.q_start[r], len = p.q_len[r];
  const int N = p.N, channels = min(CH, p.inner - c0);
  constexpr float LOG2E = 1.4426950408889634f;
  float A[PER];
#pragma unroll
  for (int i = 0; i < Q4; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = 4 * (q + SPLIT * i) + e;
      A[4 * i + e] = (active && n < N) ? -expf(p.a_log[(size_t)c * N + n]) * (FAST ? LOG2E : 1.f) : 0.f;
    }
  float* S = p.state + (size_t)p.slot_ids[r] * p.slot_stride + (size_t)(active ? c : 0) * N;
  if (N < NR || channels < CH)                           // what is never copied stays zero
    for (int i = threadIdx.x; i < 2 * BUF; i += SEL_THREADS) sel_sm[i] = 0.f;
  pdl_wait();
  const bool vec_state = (N & 3) == 0 && (p.slot_stride & 3) == 0 && ((uintptr_t)p.state & 15) == 0;
  float s[PER];
#pragma unroll
  for (int i = 0; i < Q4; ++i) {
    const int n = 4 * (q + SPLIT * i);
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (active && n < N) {
      if (vec_state) {
        v = *reinterpret_cast<const float4*>(S + n);
      } else {
        v.x = S[n];
        if (n + 1 < N) v.y = S[n + 1];
        if (n + 2 < N) v.z = S[n + 2];
        if (n + 3 < N) v.w = S[n + 3];
      }
    }
    s[4 * i] = v.x; s[4 * i + 1] = v.y; s[4 * i + 2] = v.z; s[4 * i + 3] = v.w;
  }
  __syncthreads();

  auto rows = [&](float* dst, int stride, const float* src, long long ld, int nt, int width, bool vec) {
    if (vec) {
      const int pieces = width >> 2;
      for (int i = threadIdx.x; i < nt * pieces; i += SEL_THREADS) {
        const int tt = i / pieces, c4 = i - tt * pieces;
        gb_cp_async_16(dst + tt * stride + 4 * c4, src + (size_t)tt * ld + 4 * c4);
      }
    } else {
      for (int i = threadIdx.x; i < nt * width; i += SEL_THREADS) {
        const int tt = i / width, cc = i - tt * width;
        gb_cp_async_4(dst + tt * stride + cc, src + (size_t)tt * ld + cc);
      }
    }
  };
  auto stage = [&](int t0, int b) {
    const int nt = min(TOK, len - t0);
    float* Bs = sel_sm + b * BUF;
    const size_t row0 = (size_t)(first + t0);
    rows(Bs, NR, p.B + row0 * p.ldbc, p.ldbc, nt, N, p.vec_bc);
    rows(Bs + TOK * NR, NR, p.C + row0 * p.ldbc, p.ldbc, nt, N, p.vec_bc);
    rows(Bs + 2 * TOK * NR, CH, p.x + row0 * p.ldx + c0, p.ldx, nt, channels, p.vec_x);
    rows(Bs + 2 * TOK * NR + TOK * CH, CH, p.dt + row0 * p.lddt + c0, p.lddt, nt, channels, p.vec_x);
    sel_commit();
  };

  if (len > 0) stage(0, 0);
  int b = 0;
  for (int t0 = 0; t0 < len; t0 += TOK, b ^= 1) {
    const int nt = min(TOK, len - t0);
    if (t0 + TOK < len) {
      stage(t0 + TOK, b ^ 1);
      sel_wait<1>();                                     // this chunk has landed, the next is on its way
    } else {
      sel_wait<0>();
    }
    __syncthreads();
    const float* Bs = sel_sm + b * BUF;
    const float* X = Bs + 2 * TOK * NR;
    float* Dx = sel_sm + b * BUF + 2 * TOK * NR + TOK * CH;       // raw step sizes, replaced by dt * x
    for (int i = threadIdx.x; i < nt * CH; i += SEL_THREADS) {
      const int cc = i % CH;
      if (cc < channels) {
        const float dt = hy_softplus(Dx[i] + p.dt_bias[c0 + cc]);
        sDt[i] = dt;
        Dx[i] = dt * X[i];
      } else {
        sDt[i] = 0.f;
      }
    }
    __syncthreads();
    const float* Bq = Bs + 4 * q;
    const float* Cq = Bq + TOK * NR;
    auto token = [&](int tt) {
      const float dt = sDt[tt * CH + ch], dx = Dx[tt * CH + ch];
      float y0 = 0.f, y1 = 0.f, y2 = 0.f, y3 = 0.f;      // four chains, added in a fixed order
#pragma unroll
      for (int i = 0; i < Q4; ++i) {
        const float4 b4 = *reinterpret_cast<const float4*>(Bq + tt * NR + 4 * SPLIT * i);
        const float4 c4 = *reinterpret_cast<const float4*>(Cq + tt * NR + 4 * SPLIT * i);
        const float e0 = FAST ? sel_ex2(dt * A[4 * i]) : expf(dt * A[4 * i]);
        const float e1 = FAST ? sel_ex2(dt * A[4 * i + 1]) : expf(dt * A[4 * i + 1]);
        const float e2 = FAST ? sel_ex2(dt * A[4 * i + 2]) : expf(dt * A[4 * i + 2]);
        const float e3 = FAST ? sel_ex2(dt * A[4 * i + 3]) : expf(dt * A[4 * i + 3]);
        s[4 * i] = fmaf(e0, s[4 * i], b4.x * dx);             y0 = fmaf(s[4 * i], c4.x, y0);
        s[4 * i + 1] = fmaf(e1, s[4 * i + 1], b4.y * dx);     y1 = fmaf(s[4 * i + 1], c4.y, y1);
        s[4 * i + 2] = fmaf(e2, s[4 * i + 2], b4.z * dx);     y2 = fmaf(s[4 * i + 2], c4.z, y2);
        s[4 * i + 3] = fmaf(e3, s[4 * i + 3], b4.w * dx);     y3 = fmaf(s[4 * i + 3], c4.w, y3);
      }
      return (y0 + y1) + (y2 + y3);
    };
    int tt = 0;
    for (; tt + GROUP <= nt; tt += GROUP) {
      float y[GROUP];
#pragma unroll
      for (int u = 0; u < GROUP; ++u) y[u] = token(tt + u);
      int mine = 0;
#pragma unroll
      for (int w = SPLIT / 2, carried = GROUP; w > 0; w >>= 1) {
        if (carried > 1) {
          const int half = carried / 2;
          const bool upper = q & w;
#pragma unroll
          for (int u = 0; u < GROUP / 2; ++u) {
            if (u < half) {
              const float give = upper ? y[u] : y[u + half], keep = upper ? y[u + half] : y[u];
              y[u] = keep + __shfl_xor_sync(0xffffffffu, give, w);
            }
          }
          mine += upper ? half : 0;
          carried = half;
        } else {
          y[0] += __shfl_xor_sync(0xffffffffu, y[0], w);
        }
      }
      if ((q & (SPLIT / GROUP - 1)) == 0) sY[(tt + mine) * CH + ch] = y[0];
    }
    for (; tt < nt; ++tt) {
      float y = token(tt);
#pragma unroll
      for (int w = SPLIT / 2; w > 0; w >>= 1) y += __shfl_xor_sync(0xffffffffu, y, w);
      if (q == 0) sY[tt * CH + ch] = y;
    }
    __syncthreads();
    // the chunk's outputs, neighbouring threads on neighbouring channels
    for (int i = threadIdx.x; i < nt * CH; i += SEL_THREADS) {
      const int t = i / CH, cc = i % CH;
      if (cc >= channels) continue;
      const size_t row = (size_t)(first + t0 + t);
      const float y = fmaf(p.dskip[c0 + cc], X[i], sY[i]);
      ((TO*)p.out)[row * p.ldo + c0 + cc] = from_f32<TO>(y * hy_silu(p.z[row * p.ldz + c0 + cc]));
    }
    __syncthreads();                                     // before the copies of the chunk after next land here
  }
  if (!active) return;
#pragma unroll
  for (int i = 0; i < Q4; ++i) {
    const int n = 4 * (q + SPLIT * i);
    if (n >= N) continue;
    if (vec_state) {
      *reinterpret_cast<float4*>(S + n) = make_float4(s[4 * i], s[4 * i + 1], s[4 * i + 2], s[4 * i + 3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (n + e < N) S[n + e] = s[4 * i + e];
    }
  }
}

}  // namespace

// a0 x (f32 [t, inner]), a1 its row stride, a2 raw step sizes (f32 [t, inner]), a3 their row stride, a4 B (f32 [t,
// state]), a5 C, a6 the row stride of both, a7 z (f32 [t, inner]), a8 its row stride, a9 dt_bias [inner], a10 A_log
// [inner, state], a11 D [inner], a12 state of slot 0 ([inner][state], f32), a13 elements between slots, a14 slot ids, a15
// first row per request, a16 rows per request, a17 out [t, inner], a18 its dtype (bfloat16: decays by the hardware's
// 2^x), a19 its row stride, a20 requests, a21 inner, a22 state
GB_OP(gb_op_selective_scan) {
  const int R = (int)a[20];
  if (R <= 0) return 0;
  SelParams p;
  p.x = op_ptr<const float>(a[0]); p.ldx = a[1]; p.dt = op_ptr<const float>(a[2]); p.lddt = a[3];
  p.B = op_ptr<const float>(a[4]); p.C = op_ptr<const float>(a[5]); p.ldbc = a[6];
  p.z = op_ptr<const float>(a[7]); p.ldz = a[8];
  p.dt_bias = op_ptr<const float>(a[9]); p.a_log = op_ptr<const float>(a[10]); p.dskip = op_ptr<const float>(a[11]);
  p.state = op_ptr<float>(a[12]); p.slot_stride = a[13]; p.slot_ids = op_ptr<const int>(a[14]);
  p.q_start = op_ptr<const int>(a[15]); p.q_len = op_ptr<const int>(a[16]);
  p.out = op_ptr<void>(a[17]); p.ldo = a[19];
  p.inner = (int)a[21]; p.N = (int)a[22];
  if (p.N < 1 || p.N > 256) GB_FAIL(GB_ERR_ARG, "selective_scan: %d state entries a channel (1 to 256)", p.N);
  p.vec_bc = p.N % 4 == 0 && p.ldbc % 4 == 0 && (a[4] & 15) == 0 && (a[5] & 15) == 0;
  p.vec_x = p.inner % 4 == 0 && p.ldx % 4 == 0 && p.lddt % 4 == 0 && (a[0] & 15) == 0 && (a[2] & 15) == 0;
#define SEL(SPLIT, PER, FAST, TO)                                                                                       \
  do {                                                                                                                  \
    constexpr size_t smem = sizeof(float) * SEL_TOKENS * (4 * SPLIT * PER + 6 * (SEL_THREADS / SPLIT));                 \
    static bool raised = false;            /* once, before any stream capture replays the launch */                    \
    if (!raised && smem > 48 * 1024) {                                                                                  \
      GB_CUDA((cudaFuncSetAttribute(selective_scan_kernel<SPLIT, PER, FAST, TO>,                                        \
                                    cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)));                          \
      raised = true;                                                                                                    \
    }                                                                                                                   \
    gb_launch(selective_scan_kernel<SPLIT, PER, FAST, TO>, dim3(R, gb_div_up(p.inner, SEL_THREADS / SPLIT)),             \
              dim3(SEL_THREADS), smem, ctx->stream, p);                                                                 \
  } while (0)
#define SEL_TO(SPLIT, PER) do { if (a[18] == GB_BF16) SEL(SPLIT, PER, true, bf16); else SEL(SPLIT, PER, false, float); } while (0)
  if (p.N <= 16) SEL_TO(4, 4);
  else if (p.N <= 32) SEL_TO(8, 4);
  else if (p.N <= 64) SEL_TO(16, 4);
  else if (p.N <= 128) SEL_TO(16, 8);
  else SEL_TO(32, 8);
#undef SEL_TO
#undef SEL
  GB_CHECK_LAUNCH("selective_scan");
  return 1;
}
