// What a kernel library outside this package needs in order to add an operation to the step
// plan (csrc/step_plan.cu): the signature of the operation's function, what it sees of a step,
// and the order of the step's symbols.
//
// A part with kernels of its own exports one function per operation,
//
//     extern "C" int my_op(const GbPlanCtx* ctx, const long long* a, const double* f, int flags);
//
// registers it under a name (Python: gibbs_b200.engine.plan.register_op(name, function); C:
// gb_plan_register_op) and emits records with the id it got back (PlanBuilder.emit(id, a, f,
// flags)).  When a step reaches the record, the function is called with the record's 24 integer
// operands (an operand that named a symbol holds the step's value of it: a count, or a device
// address), its 3 floating-point operands and its flags.  It launches its kernels on
// ctx->stream and returns how many it launched, or a negative number to fail the step.
// Before the call the 32-bit residual stream is whole (sums that a product had left to be added
// are added), unless the record's flags have GB_OP_TAKES_PENDING: then the function gets those sums
// (ctx->pend ...) and must itself leave the stream whole: x[m, :] += pend[0][m, :] + pend[1][m, :] + ...
// (+ pend_bias), in this order, for every row of the step.  Steps of fewer than GB_OP_PENDING_MIN_ROWS tokens are
// made whole before the call whatever the flags.
#pragma once
#include <cuda_runtime.h>

struct GbPlanCtx {
  cudaStream_t stream;
  int* status;               // the device's status word (a kernel sets it nonzero to report a failure)
  const long long* sym;      // the step's symbols, indexed by GbPlanSymbol
  int n_sym;
  // for a record whose flags have GB_OP_TAKES_PENDING (null / 0 otherwise, and when nothing is pending)
  float* residual;           // the 32-bit stream [tokens, residual_ld]
  long long residual_ld;
  const float* pend;         // [pend_splits][tokens * residual_ld] sums a product left to be added
  int pend_splits;
  const float* pend_bias;    // [residual_ld] or null
  // for a record whose flags have GB_OP_TAKES_PARTIALS (null / 0 otherwise, and when the product in front did not split
  // its sums): the partial tiles [part_splits][rows][columns] of the 32-bit output of the product recorded directly in
  // front, which was told to leave them; its output was then not written, and is their sum in this order (+ part_bias)
  const float* part;
  int part_splits;
  const float* part_bias;
};

#define GB_OP_TAKES_PENDING (1 << 30)
#define GB_OP_TAKES_PARTIALS (1 << 29)
#define GB_OP_PENDING_MIN_ROWS 64

typedef int (*GbPlanOpFn)(const GbPlanCtx* ctx, const long long* a, const double* f, int flags);

// Counts are values; the rest are device addresses of int32 arrays of the step's metadata.
enum GbPlanSymbol : int {
  GB_SYM_TOKENS = 0,         // tokens in the step
  GB_SYM_REQUESTS,           // requests in the step
  GB_SYM_WANTED,             // rows whose logits are wanted
  GB_SYM_MAX_PORTION,        // longest portion of the step
  GB_SYM_MAX_CONTEXT,        // longest context after the step (an upper bound inside CUDA graphs)
  GB_SYM_ONE_EACH,           // 1 when every request brings exactly one token
  GB_SYM_TOKEN_IDS,          // [tokens]
  GB_SYM_TOKEN_REQUEST,      // [tokens] index of the token's request within the step
  GB_SYM_TOKEN_POSITION,     // [tokens] position of the token in its request
  GB_SYM_PORTION_START,      // [requests] row of the request's first token
  GB_SYM_PORTION_LENGTH,     // [requests]
  GB_SYM_LENGTH_BEFORE,      // [requests] the request's length before the step
  GB_SYM_LENGTH_AFTER,       // [requests]
  GB_SYM_SLOT_IDS,           // [requests] state slot of the request
  GB_SYM_WANTED_ROWS,        // [wanted]
  GB_SYM_LOGITS,             // float32 [wanted, vocabulary]
  GB_SYM_BLOCK_TABLE0,       // + g (g < 15): block table of cache group g, [requests, GB_SYM_TABLE_STRIDE entries]
  GB_SYM_TABLE_STRIDE = 31,  // entries per request in this step's block tables (a value)
  GB_SYM_COUNT = 32
};
