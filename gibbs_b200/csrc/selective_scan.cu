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

constexpr int SEL_THREADS = 64, SEL_TOKENS = 16, SEL_STAGES = 4;

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
  // a long portion in segments of seg_len tokens, computed side by side (SEGMENTS below)
  int seg_len, segs;
  float* seg_state;                        // [requests][segs][inner][N]
  float* seg_time;                         // [requests][segs][inner]: the sum of a segment's step sizes
  int vec;                                 // all rows can be copied in 16-byte pieces
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
// 4 (q + SPLIT i) + e).  B, C, x, the raw step sizes and z of SEL_TOKENS tokens at a time arrive by asynchronous copies in
// a ring of SEL_STAGES buffers; what a thread copies is the same for every token, so its source and place are worked out
// once.  Tokens are taken four at a time: each lane of a channel turns ONE token's raw step size into (dt, dt x) and the
// lanes exchange them, the read-outs of the four are added over the channel's lanes together (every exchange halves what
// a lane still carries), and the lane that ends up with a token's read-out finishes it (D x, the gate).  Single tokens at
// a portion's end are computed with the same arithmetic, so how a prompt is cut does not change a bit.
//
// WHOLE: a block walks its request's whole portion.  A long prompt of one request has too few channels to fill the GPU,
// and a warp that is alone on its scheduler waits for its own latencies: the portion is then cut into segments.  ENDS
// computes, for every segment but the last, the state it leaves (from the slot's state for the first segment, from
// zero for the others) and the sum of its step sizes, without read-outs; SEGMENTS then starts every segment from
// S = S_1;  S <- exp(A time_j) S + S_j for the segments j in between, and computes read-outs.  (The first segment's
// start is copied aside by ENDS, because the last segment writes the slot.)
// FAST: exponentials of decays as the hardware's 2^x (bfloat16 models); else expf.
enum SelMode : int { WHOLE = 0, ENDS = 1, SEGMENTS = 2 };

template <int SPLIT, int PER> struct SelCfg {
  static constexpr int NR = SPLIT * PER, CH = SEL_THREADS / SPLIT;
  static constexpr int BUF = SEL_TOKENS * (2 * NR + 3 * CH);       // B [TOK][NR] | C | x [TOK][CH] | dt | z
  static constexpr int SMEM = SEL_STAGES * BUF * 4;
};

template <int SPLIT, int PER, bool FAST, typename TO, int MODE>
__global__ void __launch_bounds__(SEL_THREADS) selective_scan_kernel(SelParams p) {
  using Cf = SelCfg<SPLIT, PER>;
  constexpr int NR = Cf::NR, CH = Cf::CH, Q4 = PER / 4, TOK = SEL_TOKENS, BUF = Cf::BUF;
  static_assert(SPLIT >= 4, "four lanes share the work around four tokens");
  extern __shared__ __align__(16) float sel_sm[];        // [SEL_STAGES][BUF]
  pdl_trigger();
  const int ch = threadIdx.x / SPLIT, q = threadIdx.x % SPLIT;
  const int r = MODE == WHOLE ? blockIdx.x : blockIdx.x / p.segs, seg = MODE == WHOLE ? 0 : blockIdx.x - r * p.segs;
  const int c0 = blockIdx.y * CH, c = c0 + ch;
  const bool active = c < p.inner;
  const int all = p.q_len[r];                            // the portion
  const int first = p.q_start[r] + seg * p.seg_len;
  const int len = MODE == WHOLE ? all : min(p.seg_len, all - seg * p.seg_len);
  const bool last = MODE == WHOLE || (seg + 1) * p.seg_len >= all;
  if (len <= 0 || (MODE == ENDS && last)) {              // (nobody starts from what the last segment leaves)
    pdl_wait();                                          // a launch all of whose blocks leave still ends behind the one in front
    return;
  }
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
  const float bias = active ? p.dt_bias[c] : 0.f, dskip = active ? p.dskip[c] : 0.f;
  float* S = p.state + (size_t)p.slot_ids[r] * p.slot_stride + (size_t)(active ? c : 0) * N;
  // where segment i of this request starts from, for this channel: the slot's state (0), the state segment 0 leaves (1), or
  // what segment i - 1 leaves when it starts from zero
  const size_t seg_stride = (size_t)p.inner * N;
  float* starts = MODE == WHOLE ? nullptr : p.seg_state + (size_t)r * p.segs * seg_stride + (size_t)(active ? c : 0) * N;
  float* times = MODE == WHOLE ? nullptr : p.seg_time + (size_t)r * p.segs * p.inner + (active ? c : 0);
  if (N < NR || channels < CH)                           // what is never copied stays zero
    for (int i = threadIdx.x; i < SEL_STAGES * BUF; i += SEL_THREADS) sel_sm[i] = 0.f;
  // what this thread copies of every token: 16-byte pieces of [B | C | x | dt | z]
  constexpr int ROLES = (2 * NR / 4 + 3 * CH / 4 + SEL_THREADS - 1) / SEL_THREADS;
  const float* r_src[ROLES];
  long long r_ld[ROLES];
  int r_dst[ROLES], r_step[ROLES];
  if (p.vec) {
    const int nb = N >> 2, nx = channels >> 2;
#pragma unroll
    for (int j = 0; j < ROLES; ++j) {
      const int i = threadIdx.x + j * SEL_THREADS;
      r_src[j] = nullptr;
      r_ld[j] = 0;
      r_dst[j] = r_step[j] = 0;
      if (i < 2 * nb) {
        const int which = i / nb, c4 = 4 * (i - which * nb);
        r_ld[j] = p.ldbc;
        r_src[j] = (which ? p.C : p.B) + (size_t)first * p.ldbc + c4;
        r_dst[j] = which * TOK * NR + c4;
        r_step[j] = NR;
        if (MODE == ENDS && which == 1) r_src[j] = nullptr;        // (no read-out: no C and no z)
      } else if (i < 2 * nb + 3 * nx) {
        const int which = (i - 2 * nb) / nx, c4 = 4 * (i - 2 * nb - which * nx);
        r_ld[j] = which == 0 ? p.ldx : which == 1 ? p.lddt : p.ldz;
        r_src[j] = (which == 0 ? p.x : which == 1 ? p.dt : p.z) + (size_t)first * r_ld[j] + c0 + c4;
        r_dst[j] = 2 * TOK * NR + which * TOK * CH + c4;
        r_step[j] = CH;
        if (MODE == ENDS && which == 2) r_src[j] = nullptr;
      }
    }
  }
  pdl_wait();
  const bool vec_state = (N & 3) == 0 && (p.slot_stride & 3) == 0 && ((uintptr_t)p.state & 15) == 0;
  float s[PER] = {};
  auto fetch4 = [&](const float* src, int n) {            // entries n .. n + 3 of a channel, 0 beyond N
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (active && n < N) {
      if (vec_state) {
        v = *reinterpret_cast<const float4*>(src + n);
      } else {
        v.x = src[n];
        if (n + 1 < N) v.y = src[n + 1];
        if (n + 2 < N) v.z = src[n + 2];
        if (n + 3 < N) v.w = src[n + 3];
      }
    }
    return v;
  };
  auto store4 = [&](float* dst, int i) {
    const int n = 4 * (q + SPLIT * i);
    if (!active || n >= N) return;
    if (vec_state) {
      *reinterpret_cast<float4*>(dst + n) = make_float4(s[4 * i], s[4 * i + 1], s[4 * i + 2], s[4 * i + 3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (n + e < N) dst[n + e] = s[4 * i + e];
    }
  };
  auto decay = [&](float t, float a) { return FAST ? sel_ex2(t * a) : expf(t * a); };
#pragma unroll
  for (int i = 0; i < Q4; ++i) {
    const int n = 4 * (q + SPLIT * i);
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (MODE == WHOLE || (MODE == SEGMENTS && seg == 0 && last) || (MODE == ENDS && seg == 0)) {
      v = fetch4(S, n);
    } else if (MODE == SEGMENTS) {
      v = fetch4(starts + (seg == 0 ? 0 : seg_stride), n);
      for (int j = 2; j <= seg; ++j) {
        const float4 e = fetch4(starts + j * seg_stride, n);
        const float t = times[(size_t)(j - 1) * p.inner];
        v = make_float4(fmaf(decay(t, A[4 * i]), v.x, e.x), fmaf(decay(t, A[4 * i + 1]), v.y, e.y),
                        fmaf(decay(t, A[4 * i + 2]), v.z, e.z), fmaf(decay(t, A[4 * i + 3]), v.w, e.w));
      }
    }
    s[4 * i] = v.x; s[4 * i + 1] = v.y; s[4 * i + 2] = v.z; s[4 * i + 3] = v.w;
    if (MODE == ENDS && seg == 0) store4(starts, i);
  }
  float time = 0.f;                                      // this lane's share of the segment's step sizes
  __syncthreads();

  const int chunks = (len + TOK - 1) / TOK;
  auto stage = [&](int chunk) {                          // (always one group of copies, possibly an empty one)
    if (chunk < chunks) {
      const int t0 = chunk * TOK, nt = min(TOK, len - t0);
      float* Bs = sel_sm + (chunk % SEL_STAGES) * BUF;
      if (p.vec) {
#pragma unroll
        for (int j = 0; j < ROLES; ++j) {
          if (r_src[j] == nullptr) continue;
          const float* src = r_src[j] + (size_t)t0 * r_ld[j];
          float* dst = Bs + r_dst[j];
          if (nt == TOK) {
#pragma unroll
            for (int tt = 0; tt < TOK; ++tt, src += r_ld[j], dst += r_step[j]) gb_cp_async_16(dst, src);
          } else {
            for (int tt = 0; tt < nt; ++tt, src += r_ld[j], dst += r_step[j]) gb_cp_async_16(dst, src);
          }
        }
      } else {
        for (int tt = 0; tt < nt; ++tt) {
          const size_t row = (size_t)(first + t0 + tt);
          for (int i = threadIdx.x; i < N; i += SEL_THREADS) {
            gb_cp_async_4(Bs + tt * NR + i, p.B + row * p.ldbc + i);
            if (MODE != ENDS) gb_cp_async_4(Bs + (TOK + tt) * NR + i, p.C + row * p.ldbc + i);
          }
          float* X = Bs + 2 * TOK * NR + tt * CH;
          for (int i = threadIdx.x; i < channels; i += SEL_THREADS) {
            gb_cp_async_4(X + i, p.x + row * p.ldx + c0 + i);
            gb_cp_async_4(X + TOK * CH + i, p.dt + row * p.lddt + c0 + i);
            if (MODE != ENDS) gb_cp_async_4(X + 2 * TOK * CH + i, p.z + row * p.ldz + c0 + i);
          }
        }
      }
    }
    sel_commit();
  };

#pragma unroll
  for (int i = 0; i < SEL_STAGES - 1; ++i) stage(i);
  for (int chunk = 0; chunk < chunks; ++chunk) {
    sel_wait<SEL_STAGES - 2>();                          // this chunk's copies have landed ...
    __syncthreads();                                     // ... everybody's, and the chunk before has been used
    stage(chunk + SEL_STAGES - 1);
    const int t0 = chunk * TOK, nt = min(TOK, len - t0);
    const float* Bs = sel_sm + (chunk % SEL_STAGES) * BUF;
    const float* X = Bs + 2 * TOK * NR + ch;
    const float* Bq = Bs + 4 * q;
    const float* Cq = Bq + TOK * NR;
    auto token = [&](int tt, float dt, float dx) {
      float y0 = 0.f, y1 = 0.f, y2 = 0.f, y3 = 0.f;      // four chains, added in a fixed order
#pragma unroll
      for (int i = 0; i < Q4; ++i) {
        const float4 b4 = *reinterpret_cast<const float4*>(Bq + tt * NR + 4 * SPLIT * i);
        const float e0 = decay(dt, A[4 * i]), e1 = decay(dt, A[4 * i + 1]);
        const float e2 = decay(dt, A[4 * i + 2]), e3 = decay(dt, A[4 * i + 3]);
        if constexpr (MODE == ENDS) {
          s[4 * i] = fmaf(e0, s[4 * i], b4.x * dx);
          s[4 * i + 1] = fmaf(e1, s[4 * i + 1], b4.y * dx);
          s[4 * i + 2] = fmaf(e2, s[4 * i + 2], b4.z * dx);
          s[4 * i + 3] = fmaf(e3, s[4 * i + 3], b4.w * dx);
          continue;
        }
        const float4 c4 = *reinterpret_cast<const float4*>(Cq + tt * NR + 4 * SPLIT * i);
        s[4 * i] = fmaf(e0, s[4 * i], b4.x * dx);             y0 = fmaf(s[4 * i], c4.x, y0);
        s[4 * i + 1] = fmaf(e1, s[4 * i + 1], b4.y * dx);     y1 = fmaf(s[4 * i + 1], c4.y, y1);
        s[4 * i + 2] = fmaf(e2, s[4 * i + 2], b4.z * dx);     y2 = fmaf(s[4 * i + 2], c4.z, y2);
        s[4 * i + 3] = fmaf(e3, s[4 * i + 3], b4.w * dx);     y3 = fmaf(s[4 * i + 3], c4.w, y3);
      }
      return (y0 + y1) + (y2 + y3);
    };
    auto put = [&](int tt, float y) {
      const float xv = X[tt * CH], z = X[2 * TOK * CH + tt * CH];
      ((TO*)p.out)[(size_t)(first + t0 + tt) * p.ldo + c] = from_f32<TO>(fmaf(dskip, xv, y) * hy_silu(z));
    };
    auto four = [&](int tt) {
      const int own = tt + (q & 3);
      const float odt = hy_softplus(X[TOK * CH + own * CH] + bias), odx = odt * X[own * CH];
      float y[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float dt = __shfl_sync(0xffffffffu, odt, u, SPLIT), dx = __shfl_sync(0xffffffffu, odx, u, SPLIT);
        y[u] = token(tt + u, dt, dx);
      }
      if (MODE == ENDS) {
        time += odt;
        return;
      }
      int mine = 0;
#pragma unroll
      for (int w = SPLIT / 2, carried = 4; w > 0; w >>= 1) {
        if (carried > 1) {
          const int half = carried / 2;
          const bool upper = q & w;
#pragma unroll
          for (int u = 0; u < 2; ++u) {
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
      if (active && (q & (SPLIT / 4 - 1)) == 0) put(tt + mine, y[0]);
    };
    int tt = 0;
    if (nt == TOK) {
#pragma unroll 2
      for (; tt < TOK; tt += 4) four(tt);
    } else {
      for (; tt + 4 <= nt; tt += 4) four(tt);
    }
    for (; tt < nt; ++tt) {
      const float dt = hy_softplus(X[TOK * CH + tt * CH] + bias);
      float y = token(tt, dt, dt * X[tt * CH]);
      if (MODE == ENDS) {
        if ((q & 3) == 0) time += dt;
        continue;
      }
#pragma unroll
      for (int w = SPLIT / 2; w > 0; w >>= 1) y += __shfl_xor_sync(0xffffffffu, y, w);
      if (active && q == 0) put(tt, y);
    }
  }
  if (MODE != ENDS && !last) return;
#pragma unroll
  for (int i = 0; i < Q4; ++i) store4(MODE == ENDS ? starts + (seg + 1) * seg_stride : S, i);
  if constexpr (MODE == ENDS) {
    // (lanes q and q + 4, ... hold the same share)
    time += __shfl_xor_sync(0xffffffffu, time, 1);
    time += __shfl_xor_sync(0xffffffffu, time, 2);
    if (active && q == 0) times[(size_t)seg * p.inner] = time;
  }
}

}  // namespace

// A portion is cut into at most SEL_SEGMENTS segments of at least SEL_MIN_SEGMENT tokens, in steps of SEL_MIN_TOKENS or more.
constexpr int SEL_SEGMENTS = 8, SEL_MIN_SEGMENT = 256, SEL_MIN_TOKENS = 512;

// Floats of workspace that let up to four requests of a step have their portions cut.
GB_API long long gb_selective_scan_workspace(int inner, int state) { return 4ll * SEL_SEGMENTS * inner * (state + 1ll) + 4; }

// a0 x (f32 [t, inner]), a1 its row stride, a2 raw step sizes (f32 [t, inner]), a3 their row stride, a4 [B | C] (f32 [t,
// 2 * state]), a5 tokens, a6 the row stride of B and C, a7 z (f32 [t, inner]), a8 its row stride, a9 dt_bias [inner], a10 A_log
// [inner, state], a11 D [inner], a12 state of slot 0 ([inner][state], f32), a13 elements between slots, a14 slot ids, a15
// first row per request, a16 rows per request, a17 out [t, inner], a18 its dtype (bfloat16: decays by the hardware's
// 2^x), a19 its row stride, a20 requests, a21 inner, a22 state, a23 workspace of gb_selective_scan_workspace floats
// (16-byte aligned) or 0: portions are never cut into segments
GB_OP(gb_op_selective_scan) {
  const int R = (int)a[20];
  if (R <= 0) return 0;
  SelParams p;
  p.x = op_ptr<const float>(a[0]); p.ldx = a[1]; p.dt = op_ptr<const float>(a[2]); p.lddt = a[3];
  p.B = op_ptr<const float>(a[4]); p.C = p.B + a[22]; p.ldbc = a[6];
  p.z = op_ptr<const float>(a[7]); p.ldz = a[8];
  p.dt_bias = op_ptr<const float>(a[9]); p.a_log = op_ptr<const float>(a[10]); p.dskip = op_ptr<const float>(a[11]);
  p.state = op_ptr<float>(a[12]); p.slot_stride = a[13]; p.slot_ids = op_ptr<const int>(a[14]);
  p.q_start = op_ptr<const int>(a[15]); p.q_len = op_ptr<const int>(a[16]);
  p.out = op_ptr<void>(a[17]); p.ldo = a[19];
  p.inner = (int)a[21]; p.N = (int)a[22];
  if (p.N < 1 || p.N > 256) GB_FAIL(GB_ERR_ARG, "selective_scan: %d state entries a channel (1 to 256)", p.N);
  p.vec = p.N % 4 == 0 && p.ldbc % 4 == 0 && p.inner % 4 == 0 && p.ldx % 4 == 0 && p.lddt % 4 == 0 && p.ldz % 4 == 0 &&
          ((a[0] | a[2] | a[4] | a[7]) & 15) == 0;
  // segments: when a step of many tokens has too few channels to fill the GPU
  const int n = (int)a[5];
  const int lanes = p.N <= 16 ? 4 : p.N <= 32 ? 8 : p.N <= 128 ? 16 : 32;
  p.segs = 1; p.seg_len = 0;
  if (a[23] && n >= SEL_MIN_TOKENS && (long long)R * gb_div_up(p.inner, SEL_THREADS / lanes) < 148 * 6) {
    const int len = (gb_div_up(n, SEL_SEGMENTS) + 15) / 16 * 16;
    p.seg_len = len > SEL_MIN_SEGMENT ? len : SEL_MIN_SEGMENT;
    p.segs = gb_div_up(n, p.seg_len);
    const long long times = (long long)R * p.segs * p.inner;
    const long long floats = ((times + 3) & ~3ll) + times * p.N;
    if (floats > gb_selective_scan_workspace(p.inner, p.N)) p.segs = 1;
    p.seg_time = op_ptr<float>(a[23]);
    p.seg_state = p.seg_time + ((times + 3) & ~3ll);
  }
#define SEL_MODE(SPLIT, PER, FAST, TO, MODE)                                                                            \
  do {                                                                                                                  \
    constexpr int smem = SelCfg<SPLIT, PER>::SMEM;                                                                      \
    static bool raised = false;            /* once, before any stream capture replays the launch */                    \
    if (!raised && smem > 48 * 1024) {                                                                                  \
      GB_CUDA((cudaFuncSetAttribute(selective_scan_kernel<SPLIT, PER, FAST, TO, MODE>,                                  \
                                    cudaFuncAttributeMaxDynamicSharedMemorySize, smem)));                               \
      raised = true;                                                                                                    \
    }                                                                                                                   \
    gb_launch(selective_scan_kernel<SPLIT, PER, FAST, TO, MODE>,                                                        \
              dim3(R * p.segs, gb_div_up(p.inner, SEL_THREADS / SPLIT)), dim3(SEL_THREADS), smem, ctx->stream, p);      \
  } while (0)
#define SEL(SPLIT, PER, FAST, TO)                                                                                       \
  do {                                                                                                                  \
    if (p.segs == 1) {                                                                                                  \
      SEL_MODE(SPLIT, PER, FAST, TO, WHOLE);                                                                            \
    } else {                                                                                                            \
      SEL_MODE(SPLIT, PER, FAST, TO, ENDS);                                                                             \
      SEL_MODE(SPLIT, PER, FAST, TO, SEGMENTS);                                                                         \
    }                                                                                                                   \
  } while (0)
#define SEL_TO(SPLIT, PER) do { if (a[18] == GB_BF16) SEL(SPLIT, PER, true, bf16); else SEL(SPLIT, PER, false, float); } while (0)
  if (p.N <= 16) SEL_TO(4, 4);
  else if (p.N <= 32) SEL_TO(8, 4);
  else if (p.N <= 64) SEL_TO(16, 4);
  else if (p.N <= 128) SEL_TO(16, 8);
  else SEL_TO(32, 8);
#undef SEL_TO
#undef SEL
#undef SEL_MODE
  GB_CHECK_LAUNCH("selective_scan");
  return p.segs == 1 ? 1 : 2;
}
