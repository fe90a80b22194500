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
//  delta_chunk_scan   the chunks in order, a block per (request, head, 8 columns of S): U = U0 - W S, then S; leaves every
//                     chunk's U and the state it starts from
//  delta_chunk_read   every chunk by itself again: the read-outs, from its U and the state it starts from
#include "delta_chunks.cuh"

namespace {

constexpr int DC = DELTA_CHUNK;                          // tokens of a chunk
constexpr int PREP_THREADS = 256, SCAN_COLS = 8, READ_THREADS = 256, READ_COLS = 64;

__device__ __forceinline__ void dc_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int LEFT> __device__ __forceinline__ void dc_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(LEFT) : "memory"); }

// Request and chunk within it of chunk number `ci` of the step (r = R: there are fewer).
__device__ __forceinline__ void find_chunk(const DeltaChunkParams& p, int& r, int& ci) {
  for (r = 0; r < p.R; ++r) {
    const int c = (p.q_len[r] + DC - 1) / DC;
    if (ci < c) return;
    ci -= c;
  }
}

template <int DK>
__global__ void __launch_bounds__(PREP_THREADS, 2) delta_chunk_prep_kernel(DeltaChunkParams p) {
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
  int r, ci = blockIdx.x;
  find_chunk(p, r, ci);
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
    if (isk) {
#pragma unroll
      for (int t = 0; t < DC; ++t) x[t] = bt[t] * G[t] * ks[t * LD + c];
    } else {
      const float* v = p.qk + (size_t)row0 * p.ld_qk + p.v_col + h * p.vdim + c - p.dim;
#pragma unroll
      for (int t = 0; t < DC; ++t) x[t] = ldcg_now(v + (size_t)min(t, rows - 1) * p.ld_qk);      // (all on their way together)
#pragma unroll
      for (int t = 0; t < DC; ++t) x[t] *= bt[t];          // (0 beyond the portion)
    }
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

// A scan block's shared memory: two stages of [W | K] rows (LD floats apart), U0 and gains; S by columns; partial sums; U times
// the decays behind it, by columns.
template <int DK>
struct ScanLayout {
  static constexpr int LD = DK + 4, ULD = DC + 4, WARPS = DK / 16, THREADS = 32 * WARPS;
  static constexpr int STAGE = 2 * DC * LD + DC * SCAN_COLS + 2 * DC;
  static constexpr int S = SCAN_COLS * LD, PART = WARPS * SCAN_COLS * ULD, U = SCAN_COLS * ULD;
  static constexpr int BYTES = 4 * (2 * STAGE + S + PART + U);
};

// A thread looks after four rows of S in one column; every warp after 16 rows in the sums over rows.
template <int DK>
__global__ void __launch_bounds__(ScanLayout<DK>::THREADS) delta_chunk_scan_kernel(DeltaChunkParams p) {
  using L = ScanLayout<DK>;
  constexpr int LD = L::LD, ULD = L::ULD, WARPS = L::WARPS, THREADS = L::THREADS;
  extern __shared__ __align__(16) float dcs[];
  float* Ssm = dcs + 2 * L::STAGE;                       // [column][LD]
  float* part = Ssm + L::S;                              // [warp][column][ULD]: W S, token by token
  float* Usc = part + L::PART;                           // [column][ULD]
  pdl_trigger();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int r = blockIdx.x, h = blockIdx.y, g = h / (p.H / p.G), c0 = blockIdx.z * SCAN_COLS;
  const int first = p.q_start[r], len = p.q_len[r];
  int chunk0 = 0;                                        // number of this request's first chunk in the step
  for (int i = 0; i < r; ++i) chunk0 += (p.q_len[i] + DC - 1) / DC;
  const int vcols = min(SCAN_COLS, p.vdim - c0);         // (a multiple of four)
  // rows d .. d + 3 of column c
  constexpr int DGROUPS = DK / 32;                       // warps side by side over the rows
  const int d = 32 * (warp % DGROUPS) + 4 * (lane & 7), c = 4 * (warp / DGROUPS) + (lane >> 3);
  const bool mine = d < p.dim && c < vcols;
  float* S = p.state + (size_t)p.slot_ids[r] * p.slot_stride + ((size_t)h * p.dim + d) * p.vdim + c0 + c;
  for (int i = threadIdx.x; i < L::BYTES / 4; i += THREADS) dcs[i] = 0.f;       // what is never copied stays zero
  __syncthreads();
  pdl_wait();
  const int chunks = (len + DC - 1) / DC;
  // what this thread copies of every chunk: piece pc of rows pt, pt + PSTEP, ... of W and K, at most one piece of U0 and one gain
  constexpr int PSTEP = THREADS / (DK / 4);
  const int pt = threadIdx.x / (DK / 4), pc = 4 * (threadIdx.x % (DK / 4));
  const size_t ldw = (size_t)p.H * p.dim, ldu = (size_t)p.H * p.vdim;
  const float* wsrc = pc < p.dim ? p.w + (size_t)(first + pt) * ldw + h * p.dim + pc : nullptr;
  const float* ksrc = p.qk + (size_t)(first + pt) * p.ld_qk + p.k_col + g * p.dim + pc;
  const int ut = threadIdx.x >> 1, u4 = 4 * (threadIdx.x & 1);
  const float* usrc = p.u0 + (size_t)(first + ut) * ldu + h * p.vdim + c0 + u4;
  const float* gsrc = p.gains + ((size_t)(first + ut) * p.H + h) * 2 + (threadIdx.x & 1);
  auto stage = [&](int ci) {                             // (called with 0, 1, 2, ...: the sources move on by a chunk each time)
    if (ci < chunks) {
      float* st = dcs + (ci & 1) * L::STAGE;
      const int rows = min(DC, len - ci * DC);
      if (wsrc != nullptr) {
        float* dst = st + pt * LD + pc;
        const float* w = wsrc;
        const float* k = ksrc;
#pragma unroll
        for (int j = 0; j < DC / PSTEP; ++j) {
          if (pt + j * PSTEP < rows) {
            gb_cp_async_16(dst, w);
            gb_cp_async_16(dst + DC * LD, k);
          }
          dst += PSTEP * LD;
          w += PSTEP * ldw;
          k += PSTEP * p.ld_qk;
        }
        wsrc += DC * ldw;
        ksrc += DC * p.ld_qk;
      }
      float* u0 = st + 2 * DC * LD;
      for (int i = threadIdx.x, j = 0; i < 2 * DC; i += THREADS, j += THREADS / 2) {
        if (ut + j >= rows) continue;
        if (u4 < vcols) gb_cp_async_16(u0 + (ut + j) * SCAN_COLS + u4, usrc + j * ldu);
        gb_cp_async_4(u0 + DC * SCAN_COLS + i, gsrc + (size_t)j * p.H * 2);
      }
      usrc += DC * ldu;
      gsrc += (size_t)DC * p.H * 2;
    }
    dc_commit();
  };
  stage(0);
  float s[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) s[e] = mine ? S[(size_t)e * p.vdim] : 0.f;
  // lanes of the sums over rows: tokens tp and tp + 16, four columns from 4 ch
  const int tp = lane >> 1, ch = lane & 1;
  for (int ci = 0; ci < chunks; ++ci) {
    // the state this chunk starts from, for whoever computes the read-outs, and for this block's other threads
    const float4 s4 = make_float4(s[0], s[1], s[2], s[3]);
    *reinterpret_cast<float4*>(Ssm + c * LD + d) = s4;
    if (mine)
      *reinterpret_cast<float4*>(p.starts + (((size_t)(chunk0 + ci) * p.H + h) * p.vdim + c0 + c) * p.dim + d) = s4;
    dc_wait<0>();
    __syncthreads();                                     // this chunk's rows have landed, S stands in shared memory,
    stage(ci + 1);                                       // and the chunk before has been used
    const float* W = dcs + (ci & 1) * L::STAGE;
    const float* K = W + DC * LD;
    const float* u0 = K + DC * LD;
    const float* gr = u0 + DC * SCAN_COLS;
    const int rows = min(DC, len - ci * DC);
    {
      float acc[2][4] = {};
      const float* w0 = W + tp * LD + 16 * warp;
      const float* x0 = Ssm + 4 * ch * LD + 16 * warp;
#pragma unroll
      for (int i = 0; i < 16; i += 4) {
        const float4 a = *reinterpret_cast<const float4*>(w0 + i), b = *reinterpret_cast<const float4*>(w0 + 16 * LD + i);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float4 x = *reinterpret_cast<const float4*>(x0 + e * LD + i);
          acc[0][e] = fmaf(a.w, x.w, fmaf(a.z, x.z, fmaf(a.y, x.y, fmaf(a.x, x.x, acc[0][e]))));
          acc[1][e] = fmaf(b.w, x.w, fmaf(b.z, x.z, fmaf(b.y, x.y, fmaf(b.x, x.x, acc[1][e]))));
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float* dst = part + (warp * SCAN_COLS + 4 * ch + e) * ULD + tp;
        dst[0] = acc[0][e];
        dst[16] = acc[1][e];
      }
    }
    __syncthreads();
    // U, token `lane`, columns warp, warp + WARPS, ...
#pragma unroll
    for (int cc = warp; cc < SCAN_COLS; cc += WARPS) {
      float a = 0.f;
#pragma unroll
      for (int w = 0; w < WARPS; ++w) a += part[(w * SCAN_COLS + cc) * ULD + lane];
      const float u = lane < rows ? u0[lane * SCAN_COLS + cc] - a : 0.f;
      Usc[cc * ULD + lane] = u * gr[2 * lane + 1];
      if (cc < vcols) p.u[(((size_t)(chunk0 + ci) * p.H + h) * p.vdim + c0 + cc) * DC + lane] = u;
    }
    const float last = gr[2 * (rows - 1)];
    __syncthreads();
#pragma unroll
    for (int e = 0; e < 4; ++e) s[e] *= last;
#pragma unroll
    for (int t4 = 0; t4 < DC; t4 += 4) {
      const float4 u4 = *reinterpret_cast<const float4*>(Usc + c * ULD + t4);
      const float u[4] = {u4.x, u4.y, u4.z, u4.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float4 k = *reinterpret_cast<const float4*>(K + (t4 + i) * LD + d);
        s[0] = fmaf(k.x, u[i], s[0]); s[1] = fmaf(k.y, u[i], s[1]);
        s[2] = fmaf(k.z, u[i], s[2]); s[3] = fmaf(k.w, u[i], s[3]);
      }
    }
  }
  if (mine) {
#pragma unroll
    for (int e = 0; e < 4; ++e) S[(size_t)e * p.vdim] = s[e];
  }
}

// o_t = G_t S0^T q_t + sum_s read[t][s] u_s for one chunk, one head and READ_COLS columns; a thread two tokens and four columns.
template <int DK>
struct ReadLayout {
  static constexpr int LD = DK + 4, ULD = DC + 4;
  static constexpr int BYTES = 4 * (DC * LD + READ_COLS * LD + DC * ULD + READ_COLS * ULD + DC);
};

template <int DK>
__global__ void __launch_bounds__(READ_THREADS) delta_chunk_read_kernel(DeltaChunkParams p) {
  using L = ReadLayout<DK>;
  constexpr int LD = L::LD, ULD = L::ULD;
  extern __shared__ __align__(16) float dcr[];
  float* Q = dcr;                                        // [DC][LD]
  float* S = Q + DC * LD;                                // [column][LD]
  float* A = S + READ_COLS * LD;                         // [t][ULD]
  float* U = A + DC * ULD;                               // [column][ULD]
  float* G = U + READ_COLS * ULD;
  pdl_trigger();
  int r, ci = blockIdx.x;
  find_chunk(p, r, ci);
  pdl_wait();
  if (r == p.R) return;
  const int h = blockIdx.y, g = h / (p.H / p.G), c0 = blockIdx.z * READ_COLS;
  const int row0 = p.q_start[r] + ci * DC, rows = min(DC, p.q_len[r] - ci * DC), cols = min(READ_COLS, p.vdim - c0);
  const float* start = p.starts + (((size_t)blockIdx.x * p.H + h) * p.vdim + c0) * p.dim;
  const float* us = p.u + (((size_t)blockIdx.x * p.H + h) * p.vdim + c0) * DC;
  // (rows and columns that are not there are read from the last one that is, and what comes of them is not stored; entries
  // beyond dim are zero on both sides)
  for (int i = threadIdx.x; i < (DC + READ_COLS) * (DK / 4); i += READ_THREADS) {
    const int t = i / (DK / 4), c4 = 4 * (i % (DK / 4));
    float* dst = Q + t * LD + c4;                        // (S lies behind Q)
    if (c4 >= p.dim) *reinterpret_cast<float4*>(dst) = make_float4(0.f, 0.f, 0.f, 0.f);
    else if (t < DC) gb_cp_async_16(dst, p.qk + (size_t)(row0 + min(t, rows - 1)) * p.ld_qk + g * p.dim + c4);
    else gb_cp_async_16(dst, start + (size_t)min(t - DC, cols - 1) * p.dim + c4);
  }
  for (int i = threadIdx.x; i < (DC + READ_COLS) * (DC / 4); i += READ_THREADS) {
    const int t = i / (DC / 4), c4 = 4 * (i % (DC / 4));
    float* dst = A + t * ULD + c4;                       // (U lies behind A)
    if (t < DC) gb_cp_async_16(dst, p.read + ((size_t)(row0 + min(t, rows - 1)) * p.H + h) * DC + c4);
    else gb_cp_async_16(dst, us + (size_t)min(t - DC, cols - 1) * DC + c4);
  }
  if (threadIdx.x < DC) gb_cp_async_4(G + threadIdx.x, p.gains + ((size_t)(row0 + min((int)threadIdx.x, rows - 1)) * p.H + h) * 2);
  gb_cp_async_wait_all();
  __syncthreads();
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[2][4] = {};
  auto product = [&](const float* a, const float* b, int ld, int k) {
    const float4 a0 = *reinterpret_cast<const float4*>(a + ty * ld + k), a1 = *reinterpret_cast<const float4*>(a + (ty + 16) * ld + k);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float4 x = *reinterpret_cast<const float4*>(b + (tx + 16 * e) * ld + k);
      acc[0][e] = fmaf(a0.w, x.w, fmaf(a0.z, x.z, fmaf(a0.y, x.y, fmaf(a0.x, x.x, acc[0][e]))));
      acc[1][e] = fmaf(a1.w, x.w, fmaf(a1.z, x.z, fmaf(a1.y, x.y, fmaf(a1.x, x.x, acc[1][e]))));
    }
  };
#pragma unroll 4
  for (int k = 0; k < DK; k += 4) product(Q, S, LD, k);
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] *= G[ty + 16 * i];
#pragma unroll
  for (int k = 0; k < DC; k += 4) product(A, U, ULD, k);
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int t = ty + 16 * i;
    if (t >= rows) continue;
    float* o = p.out + (size_t)(row0 + t) * p.ldo + (size_t)h * p.vdim + c0;
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (tx + 16 * e < cols) o[tx + 16 * e] = acc[i][e];
  }
}

template <int DK>
int launch(const DeltaChunkParams& p, int n, cudaStream_t stream) {
  constexpr int prep_smem = 4 * (2 * DC * (DK + 4) + 2 * DC * (DC + 4) + 3 * DC);
  // A launch that begins while the kernel in front still runs is placed where there is room, several blocks on the SMs that
  // emptied first.  The scan lives on one SM's shared memory a block: with no more blocks than SMs it asks for so much of it that
  // two do not fit.
  constexpr int scan_alone = ScanLayout<DK>::BYTES > 120 * 1024 ? ScanLayout<DK>::BYTES : 120 * 1024;
  static bool raised = false;                            // once, before any stream capture replays the launch
  if (!raised) {
    GB_CUDA(cudaFuncSetAttribute(delta_chunk_prep_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, prep_smem));
    GB_CUDA(cudaFuncSetAttribute(delta_chunk_scan_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, scan_alone));
    GB_CUDA(cudaFuncSetAttribute(delta_chunk_read_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, ReadLayout<DK>::BYTES));
    raised = true;
  }
  const int chunks = gb_delta_chunks_count(n, p.R);
  gb_launch(delta_chunk_prep_kernel<DK>, dim3(chunks, p.H), dim3(PREP_THREADS), prep_smem, stream, p);
  GB_CHECK_LAUNCH("delta_scan (chunks by themselves)");
  const dim3 scan_grid(p.R, p.H, gb_div_up(p.vdim, SCAN_COLS));
  const int scan_smem = (long long)scan_grid.x * scan_grid.y * scan_grid.z <= 148 ? scan_alone : ScanLayout<DK>::BYTES;
  gb_launch(delta_chunk_scan_kernel<DK>, scan_grid, dim3(ScanLayout<DK>::THREADS), scan_smem, stream, p);
  GB_CHECK_LAUNCH("delta_scan (chunks in order)");
  gb_launch(delta_chunk_read_kernel<DK>, dim3(chunks, p.H, gb_div_up(p.vdim, READ_COLS)), dim3(READ_THREADS), ReadLayout<DK>::BYTES,
            stream, p);
  GB_CHECK_LAUNCH("delta_scan (read-outs)");
  return 3;
}

}  // namespace

int gb_delta_chunks(DeltaChunkParams p, float* ws, int n, cudaStream_t stream) {
  const size_t chunks = gb_delta_chunks_count(n, p.R);
  p.starts = ws;
  p.u = p.starts + chunks * p.H * p.vdim * p.dim;
  p.w = p.u + chunks * p.H * p.vdim * DC;
  p.u0 = p.w + (size_t)n * p.H * p.dim;
  p.read = p.u0 + (size_t)n * p.H * p.vdim;
  p.gains = p.read + (size_t)n * p.H * DC;
  if (p.dim <= 32) return launch<32>(p, n, stream);
  if (p.dim <= 64) return launch<64>(p, n, stream);
  return launch<128>(p, n, stream);
}
