// Attention without a softmax on the tensor cores (gated_attention_tc.cuh with SIG): the weight of a visible key is
// sigmoid(score + bias[head]), the weights are not normalised over keys, the output is multiplied by a factor.
#include "gated_attention_tc.cuh"

// operands as of gb_op_sink_attention_tc, with a23 the bias per head (f32 [heads]) or 0, no sink, no maps and no kept
// first positions; f0 scale, f1 soft cap (0: none), f2 the factor
GB_OP(gb_op_sigmoid_attention_tc) {
  return run_attention_tc<true>(ctx, a, f, flags, op_ptr<const float>(a[23]), (float)f[2]);
}
