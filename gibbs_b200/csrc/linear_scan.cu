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
//  gb_op_low_rank_decays     g = sigmoid(W z + bias)^(1 / tau) per channel, z a few entries a token: the second half of a
//                            low-rank projection and the decay in one kernel.  All in 32-bit.
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
  // a long portion in segments of seg_len tokens, computed side by side (SEGMENTS below)
  int seg_len, segs;
  float* seg_state;                        // [requests][segs][heads][cols][dim]
  float* seg_decay;                        // [requests][segs][heads * dim] or [requests][segs][heads]
  int vec_rows, vec_v;                     // rows of q, k, g (of v) can be copied in 16-byte pieces
};

__device__ __forceinline__ void ls_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int LEFT> __device__ __forceinline__ void ls_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(LEFT) : "memory");
}

// Columns of S lie in the registers of SPLIT neighbouring lanes: a lane holds PER of the dim values of CPL neighbouring
// columns (dim <= SPLIT * PER; lane q holds rows 4 (q + SPLIT i) + e), so that what it reads of q, k and g from shared
// memory, whose bandwidth is what this kernel lives on, serves CPL columns.  The inputs of TOK tokens at a time arrive by
// asynchronous copies in a ring of LS_STAGES buffers, of which all but one are on their way while one is consumed; what a
// thread copies is the same for every token, so its source and place are worked out once.  GROUP tokens are computed one
// after the other, each leaving this lane's shares of CPL read-outs in registers, and the shares of all of them are then
// added over the lanes together, every exchange halving what a lane still carries.  A portion's last tokens, fewer than
// GROUP, are added one by one in the same order of additions, so how a prompt is cut does not change a bit.
//
// WHOLE: a block walks its request's whole portion.  A long prompt of one request has too few columns to fill the GPU, and
// a warp that is alone on its scheduler waits for its own latencies: the portion is then cut into segments.  ENDS
// computes, for every segment but the last, the state it leaves (from the slot's state for the first segment, from
// zero for the others) and the product of its decays, without read-outs; SEGMENTS then starts every segment from
// S = S_1;  S <- decay_j S + S_j for the segments j in between, and computes read-outs.  (The first segment's start
// is copied aside by ENDS, because the last segment writes the slot.)
enum ScanMode : int { WHOLE = 0, ENDS = 1, SEGMENTS = 2 };
constexpr int LS_STAGES = 3, CPL = 4, GROUP = 4;

template <int SPLIT, int PER, int TOK, bool CHANNEL>
struct ScanCfg {
  static constexpr int NR = SPLIT * PER, COLS = LS_THREADS / SPLIT * CPL, ROWS = CHANNEL ? 3 : 2;
  static constexpr int BUF = TOK * (ROWS * NR + COLS + 4);   // q [TOK][NR] | k | (g) | v [TOK][COLS] | (g, w, -, -) [TOK]
  static constexpr int SMEM = LS_STAGES * BUF * 4;
};

// V values a lane carries, added over SPLIT lanes: lanes whose bit is set keep the upper half, the others the lower half, as
// long as there are halves.  Returns the index of the first value this lane ends up with (values 0 .. max(V / SPLIT, 1)
// of o); when there are more lanes than values, several lanes end up with the same one.
template <int SPLIT, int V>
__device__ __forceinline__ int ls_reduce(float (&o)[V], int q) {
  int mine = 0;
#pragma unroll
  for (int w = SPLIT / 2, carried = V; w > 0; w >>= 1) {
    if (carried > 1) {
      const int half = carried / 2;
      const bool upper = q & w;
#pragma unroll
      for (int u = 0; u < V / 2; ++u) {
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
  return mine;
}

template <int SPLIT, int PER, int TOK, bool CHANNEL, int MODE>
__global__ void __launch_bounds__(LS_THREADS) linear_scan_kernel(ScanParams p) {
  using C = ScanCfg<SPLIT, PER, TOK, CHANNEL>;
  constexpr int NR = C::NR, COLS = C::COLS, Q4 = PER / 4, ROWS = C::ROWS, BUF = C::BUF;
  extern __shared__ __align__(16) float ls_sm[];         // [LS_STAGES][BUF]
  pdl_trigger();
  const int cg = threadIdx.x / SPLIT, q = threadIdx.x % SPLIT;
  const int r = MODE == WHOLE ? blockIdx.x : blockIdx.x / p.segs, seg = MODE == WHOLE ? 0 : blockIdx.x - r * p.segs;
  const int h = blockIdx.y, c0 = blockIdx.z * COLS, c = c0 + cg * CPL;      // this lane's columns: c .. c + CPL - 1
  const int all = p.q_len[r];                            // the portion
  const int first = p.q_start[r] + seg * p.seg_len;
  const int len = MODE == WHOLE ? all : min(p.seg_len, all - seg * p.seg_len);
  const bool last = MODE == WHOLE || (seg + 1) * p.seg_len >= all;
  if (len <= 0 || (MODE == ENDS && last)) {              // (nobody starts from what the last segment leaves)
    pdl_wait();                                          // a launch all of whose blocks leave still ends behind the one in front
    return;
  }
  float* S = p.state + (size_t)p.slot_ids[r] * p.slot_stride + ((size_t)h * p.cols + c) * p.dim;
  // where segment i of this request starts from, for these columns: the slot's state (0), the state segment 0 leaves (1),
  // or what segment i - 1 leaves when it starts from zero
  const size_t seg_stride = (size_t)p.H * p.cols * p.dim;
  float* starts = MODE == WHOLE ? nullptr : p.seg_state + (size_t)r * p.segs * seg_stride + ((size_t)h * p.cols + c) * p.dim;
  const size_t decay_stride = CHANNEL ? (size_t)p.H * p.dim : (size_t)p.H;
  float* decays = MODE == WHOLE ? nullptr : p.seg_decay + (size_t)r * p.segs * decay_stride + (CHANNEL ? h * p.dim : h);
  const int vcols = max(0, min(COLS, p.vdim - c0));
  if (p.dim < NR || vcols < COLS)                        // what is never copied stays zero
    for (int i = threadIdx.x; i < LS_STAGES * BUF; i += LS_THREADS) ls_sm[i] = 0.f;
  // what this thread copies of every token: pieces of 16 bytes (of 4 where rows are not aligned) of [q | k | g | v]
  constexpr int VEC_ROLES = (ROWS * NR / 4 + COLS / 4 + LS_THREADS) / LS_THREADS;
  const float* r_src[VEC_ROLES];
  long long r_ld[VEC_ROLES];
  int r_dst[VEC_ROLES], r_step[VEC_ROLES];
  const bool vec = p.vec_rows && p.vec_v;
  if (vec) {
    const int pieces = p.dim >> 2;
#pragma unroll
    for (int j = 0; j < VEC_ROLES; ++j) {
      const int i = threadIdx.x + j * LS_THREADS;
      r_src[j] = nullptr;
      r_ld[j] = 0;
      r_dst[j] = r_step[j] = 0;
      if (i < ROWS * pieces) {
        const int which = i / pieces, c4 = 4 * (i - which * pieces);
        r_ld[j] = which == 0 ? p.ldq : which == 1 ? p.ldk : p.ldg;
        r_src[j] = (which == 0 ? p.q : which == 1 ? p.k : p.g) + (size_t)first * r_ld[j] + (size_t)h * p.dim + c4;
        r_dst[j] = which * TOK * NR + c4;
        r_step[j] = NR;
        if (MODE == ENDS && which == 0) r_src[j] = nullptr;        // (no read-out: no queries)
      } else if (i < ROWS * pieces + (vcols >> 2)) {
        const int c4 = 4 * (i - ROWS * pieces);
        r_ld[j] = p.ldv;
        r_src[j] = p.v + (size_t)first * p.ldv + (size_t)h * p.vdim + c0 + c4;
        r_dst[j] = ROWS * TOK * NR + c4;
        r_step[j] = COLS;
      }
    }
  }
  pdl_wait();
  const bool vec_state = (p.dim & 3) == 0 && (p.slot_stride & 3) == 0 && ((uintptr_t)p.state & 15) == 0;
  float s[CPL][PER] = {};
  auto fetch4 = [&](const float* src, int n) {            // entries n .. n + 3 of a column, 0 beyond dim
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (n < p.dim) {
      if (vec_state) {
        v = *reinterpret_cast<const float4*>(src + n);
      } else {
        v.x = src[n];
        if (n + 1 < p.dim) v.y = src[n + 1];
        if (n + 2 < p.dim) v.z = src[n + 2];
        if (n + 3 < p.dim) v.w = src[n + 3];
      }
    }
    return v;
  };
  auto store_state = [&](float* dst) {
#pragma unroll
    for (int e = 0; e < CPL; ++e) {
      if (c + e >= p.cols) continue;
#pragma unroll
      for (int i = 0; i < Q4; ++i) {
        const int n = 4 * (q + SPLIT * i);
        float* d = dst + (size_t)e * p.dim + n;
        if (n >= p.dim) continue;
        if (vec_state) {
          *reinterpret_cast<float4*>(d) = make_float4(s[e][4 * i], s[e][4 * i + 1], s[e][4 * i + 2], s[e][4 * i + 3]);
        } else {
#pragma unroll
          for (int x = 0; x < 4; ++x)
            if (n + x < p.dim) d[x] = s[e][4 * i + x];
        }
      }
    }
  };
  const bool from_slot = MODE == WHOLE || (MODE == SEGMENTS && seg == 0 && last) || (MODE == ENDS && seg == 0);
  if (MODE != ENDS || seg == 0) {
#pragma unroll
    for (int e = 0; e < CPL; ++e) {
      if (c + e >= p.cols) continue;
#pragma unroll
      for (int i = 0; i < Q4; ++i) {
        const int n = 4 * (q + SPLIT * i);
        const size_t at = (size_t)e * p.dim;
        float4 v;
        if (from_slot) {
          v = fetch4(S + at, n);
        } else {
          v = fetch4(starts + (seg == 0 ? 0 : seg_stride) + at, n);
          for (int j = 2; j <= seg; ++j) {
            const float4 x = fetch4(starts + j * seg_stride + at, n);
            float4 d;
            if (CHANNEL) {
              d = fetch4(decays + (j - 1) * decay_stride, n);
            } else {
              const float dh = decays[(j - 1) * decay_stride];
              d = make_float4(dh, dh, dh, dh);
            }
            v = make_float4(fmaf(d.x, v.x, x.x), fmaf(d.y, v.y, x.y), fmaf(d.z, v.z, x.z), fmaf(d.w, v.w, x.w));
          }
        }
        s[e][4 * i] = v.x; s[e][4 * i + 1] = v.y; s[e][4 * i + 2] = v.z; s[e][4 * i + 3] = v.w;
      }
    }
    if (MODE == ENDS) store_state(starts);
  }
  float prod[MODE == ENDS ? (CHANNEL ? PER : 1) : 1];      // the product of the segment's decays
#pragma unroll
  for (int i = 0; i < (int)(sizeof(prod) / sizeof(float)); ++i) prod[i] = 1.f;
  __syncthreads();

  const int chunks = (len + TOK - 1) / TOK;
  auto stage = [&](int chunk) {                          // (always one group of copies, possibly an empty one)
    if (chunk < chunks) {
      const int t0 = chunk * TOK, nt = min(TOK, len - t0);
      float* Q = ls_sm + (chunk % LS_STAGES) * BUF;
      if (vec) {
#pragma unroll
        for (int j = 0; j < VEC_ROLES; ++j) {
          if (r_src[j] == nullptr) continue;
          const float* src = r_src[j] + (size_t)t0 * r_ld[j];
          float* dst = Q + r_dst[j];
          if (nt == TOK) {
#pragma unroll
            for (int tt = 0; tt < TOK; ++tt, src += r_ld[j], dst += r_step[j]) gb_cp_async_16(dst, src);
          } else {
            for (int tt = 0; tt < nt; ++tt, src += r_ld[j], dst += r_step[j]) gb_cp_async_16(dst, src);
          }
        }
      } else {
        const size_t row0 = (size_t)(first + t0);
        for (int tt = 0; tt < nt; ++tt) {
          for (int i = threadIdx.x; i < p.dim; i += LS_THREADS) {
            if (MODE != ENDS) gb_cp_async_4(Q + tt * NR + i, p.q + (row0 + tt) * p.ldq + (size_t)h * p.dim + i);
            gb_cp_async_4(Q + (TOK + tt) * NR + i, p.k + (row0 + tt) * p.ldk + (size_t)h * p.dim + i);
            if (CHANNEL) gb_cp_async_4(Q + (2 * TOK + tt) * NR + i, p.g + (row0 + tt) * p.ldg + (size_t)h * p.dim + i);
          }
          for (int i = threadIdx.x; i < vcols; i += LS_THREADS)
            gb_cp_async_4(Q + ROWS * TOK * NR + tt * COLS + i, p.v + (row0 + tt) * p.ldv + (size_t)h * p.vdim + c0 + i);
        }
      }
      float* G = Q + TOK * (ROWS * NR + COLS);
      const int tt = LS_THREADS - 1 - threadIdx.x;         // (the last threads: the first ones copy most pieces)
      if (tt < nt) {
        const size_t row = (size_t)(first + t0 + tt);
        if (!CHANNEL) gb_cp_async_4(G + 4 * tt, p.g + row * p.ldg + h);
        if (p.w) gb_cp_async_4(G + 4 * tt + 1, p.w + row * p.ldw + h);
      }
    }
    ls_commit();
  };

#pragma unroll
  for (int i = 0; i < LS_STAGES - 1; ++i) stage(i);
  const bool weighted = p.w != nullptr;
  for (int chunk = 0; chunk < chunks; ++chunk) {
    ls_wait<LS_STAGES - 2>();                            // this chunk's copies have landed ...
    __syncthreads();                                     // ... everybody's, and the chunk before has been used
    stage(chunk + LS_STAGES - 1);
    const int t0 = chunk * TOK, nt = min(TOK, len - t0);
    const float* Q = ls_sm + (chunk % LS_STAGES) * BUF + 4 * q;
    const float* K = Q + TOK * NR;
    const float* G = K + TOK * NR;
    const float* V = ls_sm + (chunk % LS_STAGES) * BUF + ROWS * TOK * NR + cg * CPL;
    const float* GW = ls_sm + (chunk % LS_STAGES) * BUF + TOK * (ROWS * NR + COLS);
    // one token: the state's step, and this lane's shares of the read-outs
    auto token = [&](int tt, float* o) {
      const float4 v4 = *reinterpret_cast<const float4*>(V + tt * COLS);
      const float2 gw = *reinterpret_cast<const float2*>(GW + 4 * tt);
      float v[CPL] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
      for (int e = 0; e < CPL; ++e) {
        if (c + e == p.vdim) v[e] = 1.f;                   // the normaliser's column
        if (weighted) v[e] *= gw.y;
        if (MODE != ENDS) o[e] = 0.f;
      }
      if (MODE == ENDS && !CHANNEL) prod[0] *= gw.x;
#pragma unroll
      for (int i = 0; i < Q4; ++i) {
        const float4 k4 = *reinterpret_cast<const float4*>(K + tt * NR + 4 * SPLIT * i);
        float4 g4 = make_float4(gw.x, gw.x, gw.x, gw.x), q4 = g4;
        if (CHANNEL) g4 = *reinterpret_cast<const float4*>(G + tt * NR + 4 * SPLIT * i);
        if (MODE != ENDS) q4 = *reinterpret_cast<const float4*>(Q + tt * NR + 4 * SPLIT * i);
        if constexpr (MODE == ENDS && CHANNEL) {
          prod[4 * i] *= g4.x; prod[4 * i + 1] *= g4.y; prod[4 * i + 2] *= g4.z; prod[4 * i + 3] *= g4.w;
        }
#pragma unroll
        for (int e = 0; e < CPL; ++e) {
          float* se = s[e] + 4 * i;
          se[0] = fmaf(g4.x, se[0], k4.x * v[e]);
          se[1] = fmaf(g4.y, se[1], k4.y * v[e]);
          se[2] = fmaf(g4.z, se[2], k4.z * v[e]);
          se[3] = fmaf(g4.w, se[3], k4.w * v[e]);
          if (MODE != ENDS)
            o[e] = fmaf(se[3], q4.w, fmaf(se[2], q4.z, fmaf(se[1], q4.y, fmaf(se[0], q4.x, o[e]))));
        }
      }
    };
    // value number i of tokens tt ..: column i % CPL of token tt + i / CPL
    auto put = [&](int tt, int i, float o) {
      const size_t row = (size_t)(first + t0 + tt + i / CPL);
      const int cc = c + i % CPL;
      if (cc < p.vdim) p.out[row * p.ldo + (size_t)h * p.vdim + cc] = o * p.q_scale;
      else if (cc < p.cols) p.nq[row * p.H + h] = o * p.q_scale;
    };
    if constexpr (MODE == ENDS) {
      float none[CPL];
      if (nt == TOK) {
#pragma unroll 4
        for (int u = 0; u < TOK; ++u) token(u, none);
      } else {
        for (int u = 0; u < nt; ++u) token(u, none);
      }
    } else {
      int tt = 0;
#pragma unroll 1
      for (; tt + GROUP <= nt; tt += GROUP) {
        float o[GROUP * CPL];
#pragma unroll
        for (int u = 0; u < GROUP; ++u) token(tt + u, o + u * CPL);
        const int mine = ls_reduce<SPLIT, GROUP * CPL>(o, q);
        constexpr int LEFT = GROUP * CPL > SPLIT ? GROUP * CPL / SPLIT : 1;
        if (SPLIT <= GROUP * CPL || (q & (SPLIT / (GROUP * CPL) - 1)) == 0) {
#pragma unroll
          for (int i = 0; i < LEFT; ++i) put(tt, mine + i, o[i]);
        }
      }
      for (; tt < nt; ++tt) {
        float o[CPL];
        token(tt, o);
        const int mine = ls_reduce<SPLIT, CPL>(o, q);
        if ((q & (SPLIT / CPL - 1)) == 0) put(tt, mine, o[0]);
      }
    }
  }
  if (MODE != ENDS && !last) return;
  store_state(MODE == ENDS ? starts + (seg + 1) * seg_stride : S);
  if constexpr (MODE == ENDS) {
    if (c != 0) return;                                  // (one group of columns leaves the decays)
    float* d = decays + seg * decay_stride;
    if constexpr (CHANNEL) {
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int n = 4 * (q + SPLIT * (i >> 2)) + (i & 3);
        if (n < p.dim) d[n] = prod[i];
      }
    } else if (q == 0) {
      d[0] = prod[0];
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

// A thread takes one channel of LD_TOK tokens: its row of W is read once for them, z from shared memory.
constexpr int LD_TOK = 8, LD_THREADS = 128;

template <typename TW>
__global__ void __launch_bounds__(LD_THREADS)
low_rank_decays_kernel(const float* z, long long ldz, const TW* __restrict__ W, const float* __restrict__ bias, float* g,
                       long long ldg, int n, int width, int rank, float inv_tau) {
  extern __shared__ __align__(16) float zs[];                        // [rank][LD_TOK]
  pdl_trigger();
  const int c = blockIdx.x * LD_THREADS + threadIdx.x, t0 = blockIdx.y * LD_TOK;
  const float b = c < width ? bias[c] : 0.f;
  pdl_wait();
  for (int i = threadIdx.x; i < rank * LD_TOK; i += LD_THREADS) {
    const int tt = i / rank, r = i - tt * rank;
    zs[r * LD_TOK + tt] = t0 + tt < n ? z[(size_t)(t0 + tt) * ldz + r] : 0.f;
  }
  __syncthreads();
  if (c >= width) return;
  float acc[LD_TOK];
#pragma unroll
  for (int u = 0; u < LD_TOK; ++u) acc[u] = b;
  const TW* w = W + (size_t)c * rank;
#pragma unroll 8
  for (int r = 0; r < rank; ++r) {
    const float wr = to_f32(w[r]);
    const float4 a = *reinterpret_cast<const float4*>(zs + r * LD_TOK), e = *reinterpret_cast<const float4*>(zs + r * LD_TOK + 4);
    acc[0] = fmaf(wr, a.x, acc[0]); acc[1] = fmaf(wr, a.y, acc[1]); acc[2] = fmaf(wr, a.z, acc[2]); acc[3] = fmaf(wr, a.w, acc[3]);
    acc[4] = fmaf(wr, e.x, acc[4]); acc[5] = fmaf(wr, e.y, acc[5]); acc[6] = fmaf(wr, e.z, acc[6]); acc[7] = fmaf(wr, e.w, acc[7]);
  }
#pragma unroll
  for (int u = 0; u < LD_TOK; ++u) {
    // log sigmoid(x) = min(x, 0) - log1p(exp(-|x|))
    const float x = acc[u];
    if (t0 + u < n) g[(size_t)(t0 + u) * ldg + c] = expf((fminf(x, 0.f) - log1pf(expf(-fabsf(x)))) * inv_tau);
  }
}

// A block per (request, head).  m -> max(m + F, I) is closed under composition ((F1, I1) then (F2, I2) is
// (F1 + F2, max(I1 + F2, I2))), so a round of tokens, one a thread, is combined by scans over the lanes of each warp and
// then over the warps.
__global__ void exp_gates_kernel(const float* zi, long long ldi, const float* zf, long long ldf,
                                 const float* __restrict__ bi, const float* __restrict__ bf_, float* m_state,
                                 long long slot_stride, const int* slot_ids, const int* q_start, const int* q_len, float* g,
                                 float* w, float* floor_, int H, float cap) {
  __shared__ float wF[32], wI[32], s_m;
  pdl_trigger();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int r = blockIdx.x, h = blockIdx.y;
  const int first = q_start[r], len = q_len[r];
  float* ms = m_state + (size_t)slot_ids[r] * slot_stride + h;
  const float ib = bi[h], fb = bf_[h];
  pdl_wait();
  float m = *ms;
  float ni = 0.f, nf = 0.f;                              // the next round's logits, requested a round ahead
  auto fetch = [&](int t0) {
    const int t = t0 + threadIdx.x;
    if (t < len) {
      ni = zi[(size_t)(first + t) * ldi + h];
      nf = zf[(size_t)(first + t) * ldf + h];
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < len; t0 += blockDim.x) {
    const int t = t0 + threadIdx.x;
    const float ri = ni, rf = nf;
    fetch(t0 + blockDim.x);
    const bool in = t < len;
    const float i = in ? cap * tanhf((ri + ib) / cap) : -INFINITY;
    const float zz = cap * tanhf((rf + fb) / cap);
    // log sigmoid(z) = min(z, 0) - log1p(exp(-|z|))
    const float f = in ? fminf(zz, 0.f) - log1pf(expf(-fabsf(zz))) : 0.f;
    float F = f, I = i;                                  // composition of this warp's tokens up to t
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float Fp = __shfl_up_sync(0xffffffffu, F, o), Ip = __shfl_up_sync(0xffffffffu, I, o);
      if (lane >= o) {
        I = fmaxf(Ip + F, I);
        F = Fp + F;
      }
    }
    float mw = m;                                        // the maximum in front of this warp's tokens
    if (warps > 1) {
      __syncthreads();                                   // (the round before has read these)
      if (lane == 31) { wF[warp] = F; wI[warp] = I; }
      __syncthreads();
      for (int k = 0; k < warp; ++k) mw = fmaxf(mw + wF[k], wI[k]);
    }
    const float mt = fmaxf(mw + F, I);
    float before = __shfl_up_sync(0xffffffffu, mt, 1);
    if (lane == 0) before = mw;
    if (in) {
      const size_t at = (size_t)(first + t) * H + h;
      g[at] = expf(f + before - mt);
      w[at] = expf(i - mt);
      floor_[at] = expf(-mt);
    }
    m = __shfl_sync(0xffffffffu, mt, 31);                // (the last warp's is the round's)
    if (warps > 1) {
      if (threadIdx.x == blockDim.x - 1) s_m = mt;
      __syncthreads();
      m = s_m;
    }
  }
  if (threadIdx.x == 0) *ms = m;
}

}  // namespace

// A portion is cut into at most LS_SEGMENTS segments of at least LS_MIN_SEGMENT tokens, in steps of LS_MIN_TOKENS or more.
constexpr int LS_SEGMENTS = 16, LS_MIN_SEGMENT = 128, LS_MIN_TOKENS = 512;

// Floats of workspace that hold 32 segments (a step that would need more is not cut).
GB_API long long gb_linear_scan_workspace(int heads, int dim, int vdim, int normalised) {
  return 32ll * heads * ((long long)(vdim + (normalised ? 1 : 0)) * dim + dim) + 4;
}

// a0 q (f32; head h of row t at t * a1 + h * dim), a1 row stride, a2 k (likewise), a3 row stride, a4 v (f32; head h at
// h * vdim), a5 row stride, a6 decays (f32: [t, heads * dim], or [t, heads] with flag bit 0), a7 row stride, a8 write
// weights (f32 [t, heads]) or 0, a9 row stride, a10 state of slot 0 ([heads][vdim (+ 1)][dim], f32), a11 elements
// between slots, a12 slot ids, a13 first row per request, a14 rows per request, a15 out (f32 [t, heads * vdim]), a16 its
// row stride, a17 n . q out (f32 [t, heads]) or 0: no normaliser, a18 requests, a19 heads, a20 dim, a21 vdim, a22
// tokens, a23 workspace of gb_linear_scan_workspace floats (16-byte aligned) or 0: portions are never cut into segments;
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
  // segments: when a step of many tokens has too few columns to fill the GPU
  const int n = (int)a[22];
  const int lanes = p.dim <= 16 ? 4 : p.dim <= 32 ? 8 : p.dim <= 128 ? 16 : 32;
  const long long blocks = (long long)R * p.H * gb_div_up(p.cols, LS_THREADS / lanes * CPL);
  p.segs = 1; p.seg_len = 0;
  if (a[23] && n >= LS_MIN_TOKENS && blocks < 148 * 4) {
    const int wanted = gb_div_up(148 * 8, blocks);        // (about as many blocks as the GPU holds)
    const int len = (gb_div_up(n, wanted < LS_SEGMENTS ? wanted : LS_SEGMENTS) + 15) / 16 * 16;
    p.seg_len = len > LS_MIN_SEGMENT ? len : LS_MIN_SEGMENT;
    p.segs = gb_div_up(n, p.seg_len);
    const long long decays = (long long)R * p.segs * p.H * (channel ? p.dim : 1);
    const long long floats = ((decays + 3) & ~3ll) + (long long)R * p.segs * p.H * p.cols * p.dim;
    if (floats > gb_linear_scan_workspace(p.H, p.dim, p.vdim, p.nq != nullptr)) p.segs = 1;
    p.seg_decay = op_ptr<float>(a[23]);
    p.seg_state = p.seg_decay + ((decays + 3) & ~3ll);
  }
#define SCAN_MODE(SPLIT, PER, TOK, CHANNEL, MODE)                                                                      \
  do {                                                                                                                  \
    constexpr int smem = ScanCfg<SPLIT, PER, TOK, CHANNEL>::SMEM;                                                       \
    static bool raised = false;            /* once, before any stream capture replays the launch */                    \
    if (!raised && smem > 48 * 1024) {                                                                                  \
      GB_CUDA((cudaFuncSetAttribute(linear_scan_kernel<SPLIT, PER, TOK, CHANNEL, MODE>,                                 \
                                    cudaFuncAttributeMaxDynamicSharedMemorySize, smem)));                               \
      raised = true;                                                                                                    \
    }                                                                                                                   \
    gb_launch(linear_scan_kernel<SPLIT, PER, TOK, CHANNEL, MODE>,                                                       \
              dim3(R * p.segs, p.H, gb_div_up(p.cols, LS_THREADS / SPLIT * CPL)), dim3(LS_THREADS), smem, ctx->stream, p);    \
  } while (0)
#define SCAN_LAUNCH(SPLIT, PER, TOK, CHANNEL)                                                                          \
  do {                                                                                                                  \
    if (p.segs == 1) {                                                                                                  \
      SCAN_MODE(SPLIT, PER, TOK, CHANNEL, WHOLE);                                                                       \
    } else {                                                                                                            \
      SCAN_MODE(SPLIT, PER, TOK, CHANNEL, ENDS);                                                                        \
      SCAN_MODE(SPLIT, PER, TOK, CHANNEL, SEGMENTS);                                                                    \
    }                                                                                                                   \
  } while (0)
#define SCAN(SPLIT, PER, TOK)                                                                                           \
  do { if (channel) SCAN_LAUNCH(SPLIT, PER, TOK, true); else SCAN_LAUNCH(SPLIT, PER, TOK, false); } while (0)
  if (p.dim <= 16) SCAN(4, 4, 16);
  else if (p.dim <= 32) SCAN(8, 4, 16);
  else if (p.dim <= 64) SCAN(16, 4, 16);
  else if (p.dim <= 128) SCAN(16, 8, 8);
  else SCAN(32, 8, 8);
#undef SCAN
#undef SCAN_LAUNCH
#undef SCAN_MODE
  GB_CHECK_LAUNCH("linear_scan");
  return p.segs == 1 ? 1 : 2;
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
// a14 requests, a15 heads, a16 tokens; f0 cap
GB_OP(gb_op_exp_gates) {
  const int R = (int)a[14], H = (int)a[15];
  if (R <= 0) return 0;
  if (!(f[0] > 0.0)) GB_FAIL(GB_ERR_ARG, "exp_gates: a cap of %g", f[0]);
  const int threads = a[16] > 2 * R ? 256 : 32;          // (a few tokens a request: one warp)
  gb_launch(exp_gates_kernel, dim3(R, H), dim3(threads), 0, ctx->stream, op_ptr<const float>(a[0]), a[1],
            op_ptr<const float>(a[2]), a[3], op_ptr<const float>(a[4]), op_ptr<const float>(a[5]), op_ptr<float>(a[6]), a[7],
            op_ptr<const int>(a[8]), op_ptr<const int>(a[9]), op_ptr<const int>(a[10]), op_ptr<float>(a[11]),
            op_ptr<float>(a[12]), op_ptr<float>(a[13]), H, (float)f[0]);
  GB_CHECK_LAUNCH("exp_gates");
  return 1;
}

// a0 z (f32 [t, rank] at a row stride), a1 that stride, a2 W [width, rank], a3 its dtype, a4 bias [width] (f32), a5 decays
// out (f32), a6 their row stride, a7 tokens, a8 width, a9 rank; f0 tau
GB_OP(gb_op_low_rank_decays) {
  const int n = (int)a[7], width = (int)a[8], rank = (int)a[9];
  if (n <= 0) return 0;
  if (!(f[0] > 0.0)) GB_FAIL(GB_ERR_ARG, "low_rank_decays: a temperature of %g", f[0]);
  const size_t smem = sizeof(float) * LD_TOK * (size_t)rank;
  if (rank < 1 || smem > 48 * 1024) GB_FAIL(GB_ERR_ARG, "low_rank_decays: rank %d (1 to 1536)", rank);
  const dim3 grid(gb_div_up(width, LD_THREADS), gb_div_up(n, LD_TOK));
#define DECAYS(TW)                                                                                                      \
  gb_launch(low_rank_decays_kernel<TW>, grid, dim3(LD_THREADS), smem, ctx->stream, op_ptr<const float>(a[0]), a[1],      \
            op_ptr<const TW>(a[2]), op_ptr<const float>(a[4]), op_ptr<float>(a[5]), a[6], n, width, rank, (float)(1.0 / f[0]))
  if (a[3] == GB_BF16) DECAYS(bf16); else DECAYS(float);
#undef DECAYS
  GB_CHECK_LAUNCH("low_rank_decays");
  return 1;
}
