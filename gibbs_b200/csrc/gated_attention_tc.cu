// The softmax attention of gated_attention_tc.cuh as an operation.
#include "gated_attention_tc.cuh"

// Whether the tensor-core kernel takes these sizes (keys and values of 32 to 128 entries in steps of 32, up to
// 64 query heads a kv head, rows that 16-byte copies can address).
GB_API int gb_sink_attention_tc_supported(int heads, int kv_heads, int dim, int vdim) {
  if (kv_heads <= 0 || heads % kv_heads || heads / kv_heads > TC_ROWS) return 0;
  const bool dk = dim == 32 || dim == 64 || dim == 96 || dim == 128;
  const bool dv = vdim == 32 || vdim == 64 || vdim == 96 || vdim == 128;
  return dk && dv;
}

// a0 q [tokens, heads * dim] (bf16), a1 key pages, a2 value pages (bf16), a3 block table, a4 its entries per request,
// a5 page size, a6 number of pages, a7 token -> request, a8 token -> position, a9 gate logits (f32) or 0, a10 their row
// stride, a11 out [tokens, heads * vdim] (bf16), a12 its row stride, a13 tokens, a14 heads, a15 kv heads, a16 dim,
// a17 vdim, a18 window (0: every earlier position), a19 longest context of the step (an upper bound will do), a20
// workspace for partial results (gb_sink_attention_workspace_rows() rows of vdim + 2 floats) or 0, a21 requests, a22
// row of each request's first token [requests]; flags bit 0: the softmax has a sink, bit 1: out is 32-bit (else
// bfloat16), bit 2: a position sees its own block of `window` positions, counted from 0, bits 8 to 11: maps (0 means
// 1): q is [tokens, heads * maps * dim], a key row [maps * dim], out [tokens, heads * maps * vdim]; a23 a learned score
// of the sink per head (f32 [heads]) or 0: the sink's score is 0; f0 scale, f1 soft cap (0: none), f2 keep_first: a
// windowed position also sees the positions below this number
GB_OP(gb_op_sink_attention_tc) { return run_attention_tc<false>(ctx, a, f, flags, nullptr, 1.f); }
