// The gated delta rule with one decay per head, for portions of many tokens: chunks of 32 tokens at a time instead of one
// token after the other.  All in 32-bit.
//
// Within a chunk that starts from state S0, with G_t the product of the chunk's decays up to token t and P[t][s] that of
// the decays behind token s up to t (P[t][t] = 1),
//
//     u_t = beta_t (v_t - G_t S0^T k_t - sum_{s < t} P[t][s] (k_s . k_t) u_s)
//     o_t = G_t S0^T q_t + sum_{s <= t} P[t][s] (k_s . q_t) u_s
//     S   = G_last S0 + sum_s P[last][s] k_s u_s^T
//
// The u of a chunk solve a triangular system (I + A) U = diag(beta) V - (diag(beta G) K) S0, A[t][s] = beta_t P[t][s] (k_s . k_t)
// for s < t (the compact form of a product of Householder-like factors; for the delta rule: Yang et al., "Parallelizing
// Linear Transformers with the Delta Rule over Sequence Length").  With beta in (0, 1) and unit keys every entry of the
// inverse is bounded by one, so the substitution below loses no more than a few roundings.
//
//  delta_chunk_prep   every chunk by itself: the decay products (products, never quotients or differences of logarithms),
//                     (I + A)^-1 applied to both right-hand sides by forward substitution with a column a thread, and the
//                     weights of the read-out
//  delta_chunk_scan   the chunks in order, a block per (request, head, 8 columns of S): U = U0 - W S, O, S
#include "delta_chunks.cuh"

namespace {

constexpr int DC = DELTA_CHUNK;                          // tokens of a chunk
constexpr int PREP_THREADS = 256, SCAN_THREADS = 128, SCAN_COLS = 8;

__device__ __forceinline__ void dc_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int LEFT> __device__ __forceinline__ void dc_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(LEFT) : "memory"); }

template <int DK>
__global__ void __launch_bounds__(PREP_THREADS) delta_chunk_prep_kernel(DeltaChunkParams p) {
  constexpr int LD = DK + 4;                             // (rows of 8 neighbouring lanes start in different banks)
  extern __shared__ __align__(16) float dcp[];
  float* ks = dcp;                                       // [DC][LD]
  float* qs = ks + DC * LD;
  float* At = qs + DC * LD;                              // [s][t]: A[t][s]
  float* P = At + DC * (DC + 4);                         // [t][s]
  float* G = P + DC * (DC + 4);                          // [DC]
  float* bt = G + DC;
  float* gs = bt + DC;
  pdl_trigger();
  // this block's request and chunk (the launch covers the most chunks any step of so many tokens can have)
  int r = 0, ci = blockIdx.x;
  for (; r < p.R; ++r) {
    const int c = (p.q_len[r] + DC - 1) / DC;
    if (ci < c) break;
    ci -= c;
  }
  pdl_wait();                                            // (also of a block that leaves)
  if (r == p.R) return;
  const int h = blockIdx.y, g = h / (p.H / p.G);
  const int row0 = p.q_start[r] + ci * DC, rows = min(DC, p.q_len[r] - ci * DC);
  for (int i = threadIdx.x; i < DC * (DK / 4); i += PREP_THREADS) {
    const int t = i / (DK / 4), c4 = 4 * (i % (DK / 4));
    float4 k4 = make_float4(0.f, 0.f, 0.f, 0.f), q4 = k4;
    if (t < rows && c4 < p.dim) {
      const float* src = p.qk + (size_t)(row0 + t) * p.ld_qk + g * p.dim + c4;
      q4 = *reinterpret_cast<const float4*>(src);
      k4 = *reinterpret_cast<const float4*>(src + p.k_col);
    }
    *reinterpret_cast<float4*>(ks + t * LD + c4) = k4;
    *reinterpret_cast<float4*>(qs + t * LD + c4) = q4;
  }
  if (threadIdx.x < DC) {
    const int t = threadIdx.x;
    gs[t] = t < rows ? p.decay[(size_t)(row0 + t) * p.H + h] : 1.f;
    bt[t] = t < rows ? p.beta[(size_t)(row0 + t) * p.H + h] : 0.f;
  }
  __syncthreads();
  if (threadIdx.x < DC) {
    // lane s: the products behind token s; and of the chunk's decays up to token s
    const int s = threadIdx.x;
    float v = 1.f, whole = 1.f;
#pragma unroll
    for (int t = 0; t < DC; ++t) {
      if (t > s) v *= gs[t];
      if (t <= s) whole *= gs[t];
      P[t * (DC + 4) + s] = t >= s ? v : 0.f;
    }
    G[s] = whole;
  }
  __syncthreads();
  {
    // k_t . k_s and q_t . k_s for t in {ty, ty + 16}, s in {tx, tx + 16}
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float kk[2][2] = {}, qk[2][2] = {};
#pragma unroll 4
    for (int d = 0; d < DK; d += 4) {
      float4 a[2], b[2], c[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        a[i] = *reinterpret_cast<const float4*>(ks + (ty + 16 * i) * LD + d);
        b[i] = *reinterpret_cast<const float4*>(qs + (ty + 16 * i) * LD + d);
        c[i] = *reinterpret_cast<const float4*>(ks + (tx + 16 * i) * LD + d);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          kk[i][j] = fmaf(a[i].w, c[j].w, fmaf(a[i].z, c[j].z, fmaf(a[i].y, c[j].y, fmaf(a[i].x, c[j].x, kk[i][j]))));
          qk[i][j] = fmaf(b[i].w, c[j].w, fmaf(b[i].z, c[j].z, fmaf(b[i].y, c[j].y, fmaf(b[i].x, c[j].x, qk[i][j]))));
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int t = ty + 16 * i, s = tx + 16 * j;
        const float w = P[t * (DC + 4) + s];             // (0 for s > t)
        At[s * (DC + 4) + t] = s < t ? bt[t] * w * kk[i][j] : 0.f;
        if (t < rows) p.read[((size_t)(row0 + t) * p.H + h) * DC + s] = w * qk[i][j];
      }
    if (threadIdx.x < rows) {
      const int t = threadIdx.x;
      float* gr = p.gains + ((size_t)(row0 + t) * p.H + h) * 2;
      gr[0] = G[t];
      gr[1] = P[(DC - 1) * (DC + 4) + t];                // (decays behind the portion's end are 1)
    }
  }
  __syncthreads();
  // X <- (I + A)^-1 X, a column a thread: columns of diag(beta G) K, then of diag(beta) V
  for (int c = threadIdx.x; c < p.dim + p.vdim; c += PREP_THREADS) {
    float x[DC];
    const bool isk = c < p.dim;
#pragma unroll
    for (int t = 0; t < DC; ++t)
      x[t] = isk ? bt[t] * G[t] * ks[t * LD + c]
                 : t < rows ? bt[t] * p.qk[(size_t)(row0 + t) * p.ld_qk + p.v_col + h * p.vdim + c - p.dim] : 0.f;
#pragma unroll
    for (int s = 0; s < DC - 1; ++s) {
#pragma unroll
      for (int t4 = (s + 1) & ~3; t4 < DC; t4 += 4) {
        const float4 a = *reinterpret_cast<const float4*>(At + s * (DC + 4) + t4);       // (0 up to t = s)
        if (t4 > s) x[t4] = fmaf(-a.x, x[s], x[t4]);
        if (t4 + 1 > s) x[t4 + 1] = fmaf(-a.y, x[s], x[t4 + 1]);
        if (t4 + 2 > s) x[t4 + 2] = fmaf(-a.z, x[s], x[t4 + 2]);
        x[t4 + 3] = fmaf(-a.w, x[s], x[t4 + 3]);
      }
    }
    float* dst = isk ? p.w + ((size_t)row0 * p.H + h) * p.dim + c : p.u0 + ((size_t)row0 * p.H + h) * p.vdim + c - p.dim;
    const size_t ld = (size_t)p.H * (isk ? p.dim : p.vdim);
#pragma unroll
    for (int t = 0; t < DC; ++t)
      if (t < rows) dst[t * ld] = x[t];
  }
}

// Shared memory of a scan block: two stages of [W | Q | K] rows (LD floats apart), read-out weights, U0 and gains; S by columns;
// partial sums; U and U times the decay behind it.
template <int DK>
struct ScanLayout {
  static constexpr int LD = DK + 4, RLD = DC + 4;
  static constexpr int STAGE = 3 * DC * LD + DC * RLD + DC * SCAN_COLS + 2 * DC;
  static constexpr int S = SCAN_COLS * LD, PART = 2 * 4 * SCAN_COLS * DC, U = 2 * DC * SCAN_COLS;
  static constexpr int BYTES = 4 * (2 * STAGE + S + PART + U);
};

template <int DK>
__global__ void __launch_bounds__(SCAN_THREADS) delta_chunk_scan_kernel(DeltaChunkParams p) {
  using L = ScanLayout<DK>;
  constexpr int LD = L::LD, RLD = L::RLD;
  // rows of S a thread looks after (one of DK), and how many of the block's columns
  constexpr int GROUPS = SCAN_THREADS / DK, CPT = SCAN_COLS / GROUPS;
  static_assert(DK <= SCAN_THREADS && SCAN_COLS % GROUPS == 0, "a thread a row of S at least");
  extern __shared__ __align__(16) float dcs[];
  float* Ssm = dcs + 2 * L::STAGE;                       // [column][LD]
  float* part = Ssm + L::S;                              // [W S | Q S][warp][column][DC]
  float* Usm = part + L::PART;                           // [DC][SCAN_COLS]
  float* Usc = Usm + DC * SCAN_COLS;                     // the same times the decays behind the token
  pdl_trigger();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int r = blockIdx.x, h = blockIdx.y, g = h / (p.H / p.G), c0 = blockIdx.z * SCAN_COLS;
  const int first = p.q_start[r], len = p.q_len[r];
  const int vcols = min(SCAN_COLS, p.vdim - c0);         // (a multiple of four)
  const int d = threadIdx.x % DK, cg = threadIdx.x / DK * CPT;           // this thread's row and first column of S
  float* S = p.state + (size_t)p.slot_ids[r] * p.slot_stride + ((size_t)h * p.dim + d) * p.vdim + c0;
  for (int i = threadIdx.x; i < L::BYTES / 4; i += SCAN_THREADS) dcs[i] = 0.f;       // what is never copied stays zero
  __syncthreads();
  pdl_wait();
  float s[CPT];
#pragma unroll
  for (int e = 0; e < CPT; ++e) {
    s[e] = (d < p.dim && cg + e < vcols) ? S[cg + e] : 0.f;
    Ssm[(cg + e) * LD + d] = s[e];
  }
  const int chunks = (len + DC - 1) / DC;
  auto stage = [&](int ci) {
    if (ci < chunks) {
      float* st = dcs + (ci & 1) * L::STAGE;
      const int row0 = first + ci * DC, rows = min(DC, len - ci * DC);
      for (int i = threadIdx.x; i < DC * (DK / 4); i += SCAN_THREADS) {
        const int t = i / (DK / 4), c4 = 4 * (i % (DK / 4));
        if (t >= rows || c4 >= p.dim) continue;
        const float* src = p.qk + (size_t)(row0 + t) * p.ld_qk + g * p.dim + c4;
        float* dst = st + t * LD + c4;
        gb_cp_async_16(dst, p.w + ((size_t)(row0 + t) * p.H + h) * p.dim + c4);
        gb_cp_async_16(dst + DC * LD, src);
        gb_cp_async_16(dst + 2 * DC * LD, src + p.k_col);
      }
      float* rd = st + 3 * DC * LD;
      for (int i = threadIdx.x; i < DC * (DC / 4); i += SCAN_THREADS) {
        const int t = i / (DC / 4), c4 = 4 * (i % (DC / 4));
        if (t < rows) gb_cp_async_16(rd + t * RLD + c4, p.read + ((size_t)(row0 + t) * p.H + h) * DC + c4);
      }
      float* u0 = rd + DC * RLD;
      if (threadIdx.x < 2 * DC) {
        const int t = threadIdx.x >> 1, c4 = 4 * (threadIdx.x & 1);
        if (t < rows && c4 < vcols) gb_cp_async_16(u0 + t * SCAN_COLS + c4, p.u0 + ((size_t)(row0 + t) * p.H + h) * p.vdim + c0 + c4);
      } else {
        const int i = threadIdx.x - 2 * DC, t = i >> 1;
        if (t < rows) gb_cp_async_4(u0 + DC * SCAN_COLS + i, p.gains + ((size_t)(row0 + t) * p.H + h) * 2 + (i & 1));
      }
    }
    dc_commit();
  };
  stage(0);
  for (int ci = 0; ci < chunks; ++ci) {
    dc_wait<0>();
    __syncthreads();                                     // this chunk's rows have landed, S stands in shared memory,
    stage(ci + 1);                                       // and the chunk before has been used
    const float* W = dcs + (ci & 1) * L::STAGE;
    const float* Q = W + DC * LD;
    const float* K = Q + DC * LD;
    const float* rd = K + DC * LD;
    const float* u0 = rd + DC * RLD;
    const float* gr = u0 + DC * SCAN_COLS;
    const int row0 = first + ci * DC, rows = min(DC, len - ci * DC);
    {
      // lane t, this warp's quarter of the sums over d: W S and Q S for all columns
      float ws[SCAN_COLS] = {}, qs[SCAN_COLS] = {};
      const int d0 = warp * (DK / 4);
#pragma unroll
      for (int i = 0; i < DK / 4; i += 4) {
        const float4 w4 = *reinterpret_cast<const float4*>(W + lane * LD + d0 + i);
        const float4 q4 = *reinterpret_cast<const float4*>(Q + lane * LD + d0 + i);
#pragma unroll
        for (int e = 0; e < SCAN_COLS; ++e) {
          const float4 x = *reinterpret_cast<const float4*>(Ssm + e * LD + d0 + i);
          ws[e] = fmaf(w4.w, x.w, fmaf(w4.z, x.z, fmaf(w4.y, x.y, fmaf(w4.x, x.x, ws[e]))));
          qs[e] = fmaf(q4.w, x.w, fmaf(q4.z, x.z, fmaf(q4.y, x.y, fmaf(q4.x, x.x, qs[e]))));
        }
      }
#pragma unroll
      for (int e = 0; e < SCAN_COLS; ++e) {
        part[(warp * SCAN_COLS + e) * DC + lane] = ws[e];
        part[((4 + warp) * SCAN_COLS + e) * DC + lane] = qs[e];
      }
    }
    __syncthreads();
    // token `lane`, columns 2 warp and 2 warp + 1
    const float G = gr[2 * lane], behind = gr[2 * lane + 1];
    float o[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int c = 2 * warp + e;
      float a = 0.f, b = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        a += part[(w * SCAN_COLS + c) * DC + lane];
        b += part[((4 + w) * SCAN_COLS + c) * DC + lane];
      }
      const float u = lane < rows ? u0[lane * SCAN_COLS + c] - a : 0.f;
      Usm[lane * SCAN_COLS + c] = u;
      Usc[lane * SCAN_COLS + c] = u * behind;
      o[e] = G * b;
    }
    const float last = gr[2 * (rows - 1)];
    __syncthreads();
#pragma unroll
    for (int t4 = 0; t4 < DC; t4 += 4) {
      const float4 w = *reinterpret_cast<const float4*>(rd + lane * RLD + t4);
      const float wt[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 u = *reinterpret_cast<const float2*>(Usm + (t4 + i) * SCAN_COLS + 2 * warp);
        o[0] = fmaf(wt[i], u.x, o[0]);
        o[1] = fmaf(wt[i], u.y, o[1]);
      }
    }
    if (lane < rows && 2 * warp < vcols)
      *reinterpret_cast<float2*>(p.out + (size_t)(row0 + lane) * p.ldo + (size_t)h * p.vdim + c0 + 2 * warp) = make_float2(o[0], o[1]);
#pragma unroll
    for (int e = 0; e < CPT; ++e) s[e] *= last;
#pragma unroll 8
    for (int t = 0; t < DC; ++t) {
      const float k = K[t * LD + d];
      float u[CPT];
      if constexpr (CPT >= 4) {
#pragma unroll
        for (int e = 0; e < CPT; e += 4) *reinterpret_cast<float4*>(u + e) = *reinterpret_cast<const float4*>(Usc + t * SCAN_COLS + cg + e);
      } else {
#pragma unroll
        for (int e = 0; e < CPT; ++e) u[e] = Usc[t * SCAN_COLS + cg + e];
      }
#pragma unroll
      for (int e = 0; e < CPT; ++e) s[e] = fmaf(k, u[e], s[e]);
    }
#pragma unroll
    for (int e = 0; e < CPT; ++e) Ssm[(cg + e) * LD + d] = s[e];
    // (the barrier at the next chunk's start stands between these stores and their readers, and between this chunk's readers
    // and the copies that overwrite its rows)
  }
  if (d < p.dim) {
#pragma unroll
    for (int e = 0; e < CPT; ++e)
      if (cg + e < vcols) S[cg + e] = s[e];
  }
}

template <int DK>
int launch(const DeltaChunkParams& p, int n, cudaStream_t stream) {
  constexpr int prep_smem = 4 * (2 * DC * (DK + 4) + 2 * DC * (DC + 4) + 3 * DC), scan_smem = ScanLayout<DK>::BYTES;
  static bool raised = false;                            // once, before any stream capture replays the launch
  if (!raised) {
    GB_CUDA(cudaFuncSetAttribute(delta_chunk_prep_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, prep_smem));
    GB_CUDA(cudaFuncSetAttribute(delta_chunk_scan_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, scan_smem));
    raised = true;
  }
  gb_launch(delta_chunk_prep_kernel<DK>, dim3(gb_div_up(n, DC) + p.R, p.H), dim3(PREP_THREADS), prep_smem, stream, p);
  GB_CHECK_LAUNCH("delta_scan (chunks by themselves)");
  gb_launch(delta_chunk_scan_kernel<DK>, dim3(p.R, p.H, gb_div_up(p.vdim, SCAN_COLS)), dim3(SCAN_THREADS), scan_smem, stream, p);
  GB_CHECK_LAUNCH("delta_scan (chunks in order)");
  return 2;
}

}  // namespace

int gb_delta_chunks(DeltaChunkParams p, float* ws, int n, cudaStream_t stream) {
  p.w = ws;
  p.u0 = p.w + (size_t)n * p.H * p.dim;
  p.read = p.u0 + (size_t)n * p.H * p.vdim;
  p.gains = p.read + (size_t)n * p.H * DC;
  if (p.dim <= 32) return launch<32>(p, n, stream);
  if (p.dim <= 64) return launch<64>(p, n, stream);
  return launch<128>(p, n, stream);
}
