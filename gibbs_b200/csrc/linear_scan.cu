// Linear recurrences with a matrix state per head, over a ragged batch of prompt portions and single decoded
// tokens, with per-request state in slots.  Per head, token after token (S [dim, vdim], 32-bit, zero for a new request):
//
//     S <- diag(g_t) S + k_t (w_t v_t)^T,      o_t = S^T q_t * q_scale
//
// g_t is one decay per key channel or one per head, w_t an optional number per head.  With a normaliser the state has
// one more column whose value is always 1 (n <- g n + w k), read out as n . q.
//
//  gb_op_linear_scan         the recurrence
//  gb_op_forget_write_gates  what enters it when the forget gate decides what is written: per channel
//                            f = l + (1 - l) sigmoid(z + bias), g = f, k = 1 - f; and q = silu(q).  All in 32-bit.
//  gb_op_exp_gates           what enters it with exponential gates kept in range by a running maximum, per head:
//                            i = cap tanh((zi + bi) / cap), f = log sigmoid(cap tanh((zf + bf) / cap)),
//                            m_t = max(f + m_(t-1), i), g = exp(f + m_(t-1) - m_t), w = exp(i - m_t), and exp(-m_t)
//                            for the read-out; m starts at 0 and lives in the request's slot.
//
// State layout in a slot: [heads][vdim (+ 1)][dim]; m: [heads].
#include "hybrid.cuh"

namespace {

constexpr int LS_THREADS = 64;

struct ScanParams {
  const float* q; long long ldq;
  const float* k; long long ldk;
  const float* v; long long ldv;
  const float* g; long long ldg;           // [t, heads * dim] or [t, heads]
  const float* w; long long ldw;           // [t, heads] or null
  float* state; long long slot_stride;
  const int* slot_ids; const int* q_start; const int* q_len;
  float* out; long long ldo;
  float* nq;                               // [t, heads]: n . q * q_scale, or null: no normaliser
  int H, dim, vdim, cols;                  // cols: vdim, or vdim + 1 with the normaliser
  float q_scale;
  int vec_rows, vec_v;                     // rows of q, k, g (of v) can be copied in 16-byte pieces
};

__device__ __forceinline__ void ls_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int LEFT> __device__ __forceinline__ void ls_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(LEFT) : "memory");
}

// A column of S lies in the registers of SPLIT neighbouring lanes, PER of its dim values each (dim <= SPLIT * PER;
// lane q holds rows 4 (q + SPLIT i) + e).  The inputs of TOK tokens at a time arrive by asynchronous copies into one
// of two buffers while the tokens of the other are consumed.  GROUP tokens are computed one after the other, each
// leaving this lane's share of its read-out in a register, and the shares of all of them are then added over the lanes
// together, every exchange halving what a lane still carries: one shuffle a token instead of log2(SPLIT).  A portion's
// last tokens, fewer than GROUP, are added one by one in the same order of additions, so how a prompt is cut does not
// change a bit.
template <int SPLIT, int PER, int TOK, bool CHANNEL>
__global__ void __launch_bounds__(LS_THREADS) linear_scan_kernel(ScanParams p) {
  constexpr int NR = SPLIT * PER, COLS = LS_THREADS / SPLIT, Q4 = PER / 4;
  constexpr int GROUP = SPLIT < 8 ? SPLIT : 8;
  constexpr int ROWS = CHANNEL ? 3 : 2;
  constexpr int BUF = TOK * (ROWS * NR + COLS + 2);      // q [TOK][NR] | k | (g) | v [TOK][COLS] | g [TOK] | w [TOK]
  extern __shared__ __align__(16) float ls_sm[];         // [2][BUF]
  pdl_trigger();
  const int col = threadIdx.x / SPLIT, q = threadIdx.x % SPLIT;
  const int r = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * COLS, c = c0 + col;
  const bool active = c < p.cols;
  const bool counts = c == p.vdim;                       // the normaliser's column: its value is always 1
  const int first = p.q_start[r], len = p.q_len[r];
  float* S = p.state + (size_t)p.slot_ids[r] * p.slot_stride + ((size_t)h * p.cols + (active ? c : 0)) * p.dim;
  if (p.dim < NR || p.vdim - c0 < COLS)                  // what is never copied stays zero
    for (int i = threadIdx.x; i < 2 * BUF; i += LS_THREADS) ls_sm[i] = 0.f;
  pdl_wait();
  const bool vec_state = (p.dim & 3) == 0 && (p.slot_stride & 3) == 0 && ((uintptr_t)p.state & 15) == 0;
  float s[PER];
#pragma unroll
  for (int i = 0; i < Q4; ++i) {
    const int n = 4 * (q + SPLIT * i);
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (active && n < p.dim) {
      if (vec_state) {
        v = *reinterpret_cast<const float4*>(S + n);
      } else {
        v.x = S[n];
        if (n + 1 < p.dim) v.y = S[n + 1];
        if (n + 2 < p.dim) v.z = S[n + 2];
        if (n + 3 < p.dim) v.w = S[n + 3];
      }
    }
    s[4 * i] = v.x; s[4 * i + 1] = v.y; s[4 * i + 2] = v.z; s[4 * i + 3] = v.w;
  }
  __syncthreads();

  const int vcols = max(0, min(COLS, p.vdim - c0));
  auto stage = [&](int t0, int b) {
    const int nt = min(TOK, len - t0);
    float* Q = ls_sm + b * BUF;
    float* V = Q + ROWS * TOK * NR;
    const size_t row0 = (size_t)(first + t0);
    const float* src[3] = {p.q + row0 * p.ldq + (size_t)h * p.dim, p.k + row0 * p.ldk + (size_t)h * p.dim,
                           CHANNEL ? p.g + row0 * p.ldg + (size_t)h * p.dim : nullptr};
    const long long ld[3] = {p.ldq, p.ldk, p.ldg};
    if (p.vec_rows) {
      const int pieces = p.dim >> 2;
      for (int i = threadIdx.x; i < pieces; i += LS_THREADS) {      // (a thread's piece is the same for every token)
#pragma unroll
        for (int a = 0; a < ROWS; ++a)
          for (int tt = 0; tt < nt; ++tt)
            gb_cp_async_16(Q + (a * TOK + tt) * NR + 4 * i, src[a] + (size_t)tt * ld[a] + 4 * i);
      }
    } else {
      for (int i = threadIdx.x; i < p.dim; i += LS_THREADS)
#pragma unroll
        for (int a = 0; a < ROWS; ++a)
          for (int tt = 0; tt < nt; ++tt) gb_cp_async_4(Q + (a * TOK + tt) * NR + i, src[a] + (size_t)tt * ld[a] + i);
    }
    const float* vs = p.v + row0 * p.ldv + (size_t)h * p.vdim + c0;
    if (p.vec_v) {
      const int vp = vcols >> 2;
      for (int i = LS_THREADS - 1 - threadIdx.x; i < nt * vp; i += LS_THREADS) {
        const int tt = i / vp, c4 = i - tt * vp;
        gb_cp_async_16(V + tt * COLS + 4 * c4, vs + (size_t)tt * p.ldv + 4 * c4);
      }
    } else {
      for (int i = LS_THREADS - 1 - threadIdx.x; i < nt * vcols; i += LS_THREADS) {
        const int tt = i / vcols, cc = i - tt * vcols;
        gb_cp_async_4(V + tt * COLS + cc, vs + (size_t)tt * p.ldv + cc);
      }
    }
    float* G = V + TOK * COLS;
    if ((int)threadIdx.x < nt) {
      if (!CHANNEL) gb_cp_async_4(G + threadIdx.x, p.g + (row0 + threadIdx.x) * p.ldg + h);
      if (p.w) gb_cp_async_4(G + TOK + threadIdx.x, p.w + (row0 + threadIdx.x) * p.ldw + h);
    }
    ls_commit();
  };

  if (len > 0) stage(0, 0);
  int b = 0;
  for (int t0 = 0; t0 < len; t0 += TOK, b ^= 1) {
    const int nt = min(TOK, len - t0);
    if (t0 + TOK < len) {
      stage(t0 + TOK, b ^ 1);
      ls_wait<1>();                                      // this chunk has landed, the next is on its way
    } else {
      ls_wait<0>();
    }
    __syncthreads();
    const float* Q = ls_sm + b * BUF + 4 * q;
    const float* K = Q + TOK * NR;
    const float* G = K + TOK * NR;
    const float* V = ls_sm + b * BUF + ROWS * TOK * NR;
    const float* Gh = V + TOK * COLS;
    const float* Wh = Gh + TOK;
    // one token: the state's step, and this lane's share of the read-out
    auto token = [&](int tt) {
      float v = counts ? 1.f : V[tt * COLS + col];
      if (p.w) v *= Wh[tt];
      const float gh = CHANNEL ? 0.f : Gh[tt];
      float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;      // four chains, added in a fixed order
#pragma unroll
      for (int i = 0; i < Q4; ++i) {
        const float4 k4 = *reinterpret_cast<const float4*>(K + tt * NR + 4 * SPLIT * i);
        const float4 q4 = *reinterpret_cast<const float4*>(Q + tt * NR + 4 * SPLIT * i);
        float4 g4 = make_float4(gh, gh, gh, gh);
        if (CHANNEL) g4 = *reinterpret_cast<const float4*>(G + tt * NR + 4 * SPLIT * i);
        s[4 * i] = fmaf(g4.x, s[4 * i], k4.x * v);             d0 = fmaf(s[4 * i], q4.x, d0);
        s[4 * i + 1] = fmaf(g4.y, s[4 * i + 1], k4.y * v);     d1 = fmaf(s[4 * i + 1], q4.y, d1);
        s[4 * i + 2] = fmaf(g4.z, s[4 * i + 2], k4.z * v);     d2 = fmaf(s[4 * i + 2], q4.z, d2);
        s[4 * i + 3] = fmaf(g4.w, s[4 * i + 3], k4.w * v);     d3 = fmaf(s[4 * i + 3], q4.w, d3);
      }
      return (d0 + d1) + (d2 + d3);
    };
    auto put = [&](int tt, float o) {
      const size_t row = (size_t)(first + t0 + tt);
      if (counts) p.nq[row * p.H + h] = o * p.q_scale;
      else p.out[row * p.ldo + (size_t)h * p.vdim + c] = o * p.q_scale;
    };
    int tt = 0;
    for (; tt + GROUP <= nt; tt += GROUP) {
      float o[GROUP];
#pragma unroll
      for (int u = 0; u < GROUP; ++u) o[u] = token(tt + u);
      // lanes whose bit `w` is set keep the upper half of the tokens they carry, the others the lower half
      int mine = 0;
#pragma unroll
      for (int w = SPLIT / 2, carried = GROUP; w > 0; w >>= 1) {
        if (carried > 1) {
          const int half = carried / 2;
          const bool upper = q & w;
#pragma unroll
          for (int u = 0; u < GROUP / 2; ++u) {
            if (u < half) {
              const float give = upper ? o[u] : o[u + half], keep = upper ? o[u + half] : o[u];
              o[u] = keep + __shfl_xor_sync(0xffffffffu, give, w);
            }
          }
          mine += upper ? half : 0;
          carried = half;
        } else {
          o[0] += __shfl_xor_sync(0xffffffffu, o[0], w);
        }
      }
      // (several lanes carry the same token when there are more lanes than tokens: the first of them stores)
      if (active && (q & (SPLIT / GROUP - 1)) == 0) put(tt + mine, o[0]);
    }
    for (; tt < nt; ++tt) {
      float o = token(tt);
#pragma unroll
      for (int w = SPLIT / 2; w > 0; w >>= 1) o += __shfl_xor_sync(0xffffffffu, o, w);
      if (active && q == 0) put(tt, o);
    }
    __syncthreads();                                     // before the copies of the chunk after next land here
  }
  if (!active) return;
#pragma unroll
  for (int i = 0; i < Q4; ++i) {
    const int n = 4 * (q + SPLIT * i);
    if (n >= p.dim) continue;
    if (vec_state) {
      *reinterpret_cast<float4*>(S + n) = make_float4(s[4 * i], s[4 * i + 1], s[4 * i + 2], s[4 * i + 3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (n + e < p.dim) S[n + e] = s[4 * i + e];
    }
  }
}

// one thread an entry of [tokens, width]
__global__ void forget_write_gates_kernel(float* q, long long ldq, float* f, long long ldf, const float* __restrict__ bias,
                                          const float* __restrict__ lower, float* k, long long ldk, int n, int width) {
  pdl_trigger();
  pdl_wait();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)n * width) return;
  const int t = (int)(i / width), c = (int)(i - (long long)t * width);
  float* qp = q + (size_t)t * ldq + c;
  float* fp = f + (size_t)t * ldf + c;
  const float l = lower[c], z = *fp + bias[c];
  *qp = hy_silu(*qp);
  *fp = fmaf(1.f - l, hy_sigmoid(z), l);
  k[(size_t)t * ldk + c] = (1.f - l) * hy_sigmoid(-z);   // (1 - f without the cancellation where f is near one)
}

// One warp per (request, head).  m -> max(m + F, I) is closed under composition ((F1, I1) then (F2, I2) is
// (F1 + F2, max(I1 + F2, I2))), so 32 tokens are combined by a scan over the lanes.
__global__ void exp_gates_kernel(const float* zi, long long ldi, const float* zf, long long ldf,
                                 const float* __restrict__ bi, const float* __restrict__ bf_, float* m_state,
                                 long long slot_stride, const int* slot_ids, const int* q_start, const int* q_len, float* g,
                                 float* w, float* floor_, int H, float cap) {
  pdl_trigger();
  const int lane = threadIdx.x & 31;
  const int h = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (h >= H) return;                                    // (whole warps; nothing below meets the block)
  const int r = blockIdx.x;
  const int first = q_start[r], len = q_len[r];
  float* ms = m_state + (size_t)slot_ids[r] * slot_stride + h;
  const float ib = bi[h], fb = bf_[h];
  pdl_wait();
  float m = *ms;
  float ni = 0.f, nf = 0.f;                              // the next 32 tokens' logits, requested a round ahead
  auto fetch = [&](int t0) {
    const int t = t0 + lane;
    if (t < len) {
      ni = zi[(size_t)(first + t) * ldi + h];
      nf = zf[(size_t)(first + t) * ldf + h];
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < len; t0 += 32) {
    const int t = t0 + lane;
    const float ri = ni, rf = nf;
    fetch(t0 + 32);
    const bool in = t < len;
    const float i = in ? cap * tanhf((ri + ib) / cap) : -INFINITY;
    const float zz = cap * tanhf((rf + fb) / cap);
    // log sigmoid(z) = min(z, 0) - log1p(exp(-|z|))
    const float f = in ? fminf(zz, 0.f) - log1pf(expf(-fabsf(zz))) : 0.f;
    float F = f, I = i;                                  // composition of tokens t0 .. t
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float Fp = __shfl_up_sync(0xffffffffu, F, o), Ip = __shfl_up_sync(0xffffffffu, I, o);
      if (lane >= o) {
        I = fmaxf(Ip + F, I);
        F = Fp + F;
      }
    }
    const float mt = fmaxf(m + F, I);
    float before = __shfl_up_sync(0xffffffffu, mt, 1);
    if (lane == 0) before = m;
    if (in) {
      const size_t at = (size_t)(first + t) * H + h;
      g[at] = expf(f + before - mt);
      w[at] = expf(i - mt);
      floor_[at] = expf(-mt);
    }
    m = __shfl_sync(0xffffffffu, mt, 31);
  }
  if (lane == 0) *ms = m;
}

}  // namespace

// a0 q (f32; head h of row t at t * a1 + h * dim), a1 row stride, a2 k (likewise), a3 row stride, a4 v (f32; head h at
// h * vdim), a5 row stride, a6 decays (f32: [t, heads * dim], or [t, heads] with flag bit 0), a7 row stride, a8 write
// weights (f32 [t, heads]) or 0, a9 row stride, a10 state of slot 0 ([heads][vdim (+ 1)][dim], f32), a11 elements
// between slots, a12 slot ids, a13 first row per request, a14 rows per request, a15 out (f32 [t, heads * vdim]), a16 its
// row stride, a17 n . q out (f32 [t, heads]) or 0: no normaliser, a18 requests, a19 heads, a20 dim, a21 vdim;
// f0 factor on the read-out; flags bit 0: one decay a head
GB_OP(gb_op_linear_scan) {
  ScanParams p;
  p.q = op_ptr<const float>(a[0]); p.ldq = a[1]; p.k = op_ptr<const float>(a[2]); p.ldk = a[3];
  p.v = op_ptr<const float>(a[4]); p.ldv = a[5]; p.g = op_ptr<const float>(a[6]); p.ldg = a[7];
  p.w = op_ptr<const float>(a[8]); p.ldw = a[9]; p.state = op_ptr<float>(a[10]); p.slot_stride = a[11];
  p.slot_ids = op_ptr<const int>(a[12]); p.q_start = op_ptr<const int>(a[13]); p.q_len = op_ptr<const int>(a[14]);
  p.out = op_ptr<float>(a[15]); p.ldo = a[16]; p.nq = op_ptr<float>(a[17]);
  const int R = (int)a[18];
  p.H = (int)a[19]; p.dim = (int)a[20]; p.vdim = (int)a[21];
  p.cols = p.vdim + (p.nq ? 1 : 0);
  p.q_scale = (float)f[0];
  if (R <= 0) return 0;
  const bool channel = !(flags & 1);
  if (p.dim < 1 || p.dim > 256) GB_FAIL(GB_ERR_ARG, "linear_scan: keys of %d entries (at most 256)", p.dim);
  p.vec_rows = p.dim % 4 == 0 && p.ldq % 4 == 0 && p.ldk % 4 == 0 && (a[0] & 15) == 0 && (a[2] & 15) == 0 &&
               (!channel || (p.ldg % 4 == 0 && (a[6] & 15) == 0));
  p.vec_v = p.vdim % 4 == 0 && p.ldv % 4 == 0 && (a[4] & 15) == 0;
#define SCAN(SPLIT, PER, TOK)                                                                                           \
  do {                                                                                                                  \
    const dim3 grid(R, p.H, gb_div_up(p.cols, LS_THREADS / SPLIT));                                                     \
    const size_t smem = sizeof(float) * 2 * (size_t)TOK * ((channel ? 3 : 2) * SPLIT * PER + LS_THREADS / SPLIT + 2);   \
    if (channel) gb_launch(linear_scan_kernel<SPLIT, PER, TOK, true>, grid, dim3(LS_THREADS), smem, ctx->stream, p);    \
    else gb_launch(linear_scan_kernel<SPLIT, PER, TOK, false>, grid, dim3(LS_THREADS), smem, ctx->stream, p);           \
  } while (0)
  if (p.dim <= 16) SCAN(4, 4, 16);
  else if (p.dim <= 32) SCAN(8, 4, 16);
  else if (p.dim <= 64) SCAN(16, 4, 16);
  else if (p.dim <= 128) SCAN(8, 16, 8);
  else SCAN(16, 16, 4);                      // (a group of eight tokens never fills: added one by one)
#undef SCAN
  GB_CHECK_LAUNCH("linear_scan");
  return 1;
}

// a0 q (f32, changed in place), a1 its row stride, a2 gate logits (f32, replaced by the decays), a3 their row stride, a4
// bias [width], a5 lower bounds [width], a6 k out (f32), a7 its row stride, a8 tokens, a9 width
GB_OP(gb_op_forget_write_gates) {
  const int n = (int)a[8], width = (int)a[9];
  if (n <= 0) return 0;
  gb_launch(forget_write_gates_kernel, dim3(gb_div_up((long long)n * width, 256)), dim3(256), 0, ctx->stream,
            op_ptr<float>(a[0]), a[1], op_ptr<float>(a[2]), a[3], op_ptr<const float>(a[4]), op_ptr<const float>(a[5]),
            op_ptr<float>(a[6]), a[7], n, width);
  GB_CHECK_LAUNCH("forget_write_gates");
  return 1;
}

// a0 input-gate logits (f32 [t, heads] at a row stride), a1 that stride, a2 forget-gate logits, a3 their stride, a4 bias
// of the former [heads], a5 of the latter, a6 m of slot 0 ([heads], f32), a7 elements between slots, a8 slot ids, a9
// first row per request, a10 rows per request, a11 decays out (f32 [t, heads]), a12 write weights out, a13 exp(-m) out,
// a14 requests, a15 heads; f0 cap
GB_OP(gb_op_exp_gates) {
  const int R = (int)a[14], H = (int)a[15];
  if (R <= 0) return 0;
  if (!(f[0] > 0.0)) GB_FAIL(GB_ERR_ARG, "exp_gates: a cap of %g", f[0]);
  const int warps = H < 4 ? H : 4;
  gb_launch(exp_gates_kernel, dim3(R, gb_div_up(H, warps)), dim3(32 * warps), 0, ctx->stream, op_ptr<const float>(a[0]), a[1],
            op_ptr<const float>(a[2]), a[3], op_ptr<const float>(a[4]), op_ptr<const float>(a[5]), op_ptr<float>(a[6]), a[7],
            op_ptr<const int>(a[8]), op_ptr<const int>(a[9]), op_ptr<const int>(a[10]), op_ptr<float>(a[11]),
            op_ptr<float>(a[12]), op_ptr<float>(a[13]), H, (float)f[0]);
  GB_CHECK_LAUNCH("exp_gates");
  return 1;
}
