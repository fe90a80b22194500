// The chunked form of the delta rule's recurrence (delta_chunks.cu), launched by gb_op_delta_scan.
#pragma once
#include "hybrid.cuh"

constexpr int DELTA_CHUNK = 32;
constexpr int DELTA_CHUNK_MAX_DIM = 128;

struct DeltaChunkParams {
  const float* qk; long long ld_qk;        // rows [q | k | v]: q and k normed per key head
  int k_col, v_col;
  const float* decay;                      // [t, heads]
  const float* beta;                       // [t, heads]
  float* state; long long slot_stride;     // slot 0: [heads][dim][vdim]
  const int* slot_ids; const int* q_start; const int* q_len;
  float* out; long long ldo;               // [t, heads * vdim]
  int R, H, G, dim, vdim;
  // workspace, set by gb_delta_chunks
  float* starts;                           // [chunk of the step, heads, vdim, dim]: the state a chunk starts from
  float* u;                                // [chunk of the step, heads, vdim, DELTA_CHUNK]
  float* w;                                // [t, heads, dim]
  float* u0;                               // [t, heads, vdim]
  float* read;                             // [t, heads, DELTA_CHUNK]
  float* gains;                            // [t, heads, 2]: product of the chunk's decays up to t, and behind it
};

// The most chunks a step of n tokens in R portions has.
static inline int gb_delta_chunks_count(int n, int R) { return gb_div_up(n, DELTA_CHUNK) + R; }
// Floats of workspace for such a step.
static inline long long gb_delta_chunks_floats(int n, int R, int heads, int dim, int vdim) {
  return (long long)heads * ((long long)gb_delta_chunks_count(n, R) * vdim * (dim + DELTA_CHUNK) +
                             (long long)n * (dim + vdim + DELTA_CHUNK + 2));
}

// Rows of 16-byte pieces (dim, vdim and every column and stride a multiple of four), dim at most DELTA_CHUNK_MAX_DIM; n tokens.
// Returns the number of launches or an error.
int gb_delta_chunks(DeltaChunkParams p, float* ws, int n, cudaStream_t stream);
