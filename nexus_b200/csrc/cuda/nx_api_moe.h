// C ABI of the MoE routing kernels.
#pragma once
#include "nx_api.h"
#include "nx_api_mixers.h"

#ifdef __cplusplus
extern "C" {
#endif

// logits: FP32 [tokens, experts].  expert / gate: [tokens, k]; gate = softmax over the k selected logits;
// ties go to the lower expert id.
int nx_moe_topk(const float* logits, int tokens, int experts, int k, int32_t* expert, float* gate, nx_stream_t stream);
// slot[t, j] = position of the assignment inside its expert's buffer in priority order (j, then t), or -1
// beyond `capacity`; counts[e] = rows kept by expert e; *dropped += assignments dropped (may be null).
int nx_moe_assign(const int32_t* expert, int tokens, int k, int experts, int capacity, int32_t* slot, int32_t* counts,
                  int32_t* dropped, nx_stream_t stream);
// Capacity per group of tokens (`tokens / groups` consecutive tokens each) and the Reroute overflow policy.  The
// assignments of a group are visited in priority order (j, then t).  `order` null: an assignment past its expert's
// capacity is dropped (slot -1).  `order` [tokens, experts] (each token's experts by descending score): such an
// assignment moves to the token's best expert that has room and is none of its own choices (`expert` is updated in
// place, *rerouted counts them) and is dropped only when there is none.  slot = group * capacity + position, i.e.
// the expert buffers are [experts, groups * capacity, d]; counts[g * experts + e] = rows of group g kept by expert e.
int nx_moe_assign_groups(int32_t* expert, const int32_t* order, int tokens, int k, int experts, int groups,
                         int capacity, int32_t* slot, int32_t* counts, int32_t* dropped, int32_t* rerouted,
                         nx_stream_t stream);
// dgate[t, j] = dy[t] . expert_out[expert[t,j]][slot[t,j]]  (BF16 rows of d elements)
int nx_moe_gate_grad(const void* dy, const void* expert_out, const int32_t* expert, const int32_t* slot, float* dgate,
                     int tokens, int k, int d, int capacity, nx_stream_t stream);


// Experts by token id, for all layers of a step in one launch.  Layer l: table [vocab, top] gives every token's experts;
// its assignments (token t, choice j) are sorted by expert, every expert's slots starting at a multiple of `align`:
//   slots[t * top + j]   slot of the assignment          rows[slot]    its token, -1 between the experts
//   start[e], count[e]   first slot and number of slots  groups[slot / align]   expert, -1 past the last one
// The order of one expert's assignments among themselves is not fixed.  max_slots is a multiple of align and at least
// moe_table_slots(tokens * top, experts, align).
#define NX_TABLE_LAYERS 32
typedef struct NxTableRouteLayer {
  const int32_t* table;
  int32_t* slots;
  int32_t* rows;
  int32_t* start;
  int32_t* count;
  int32_t* groups;
  int32_t experts, top, max_slots;
} NxTableRouteLayer;
typedef struct NxTableRouteArgs {
  const int32_t* tokens;
  int32_t n, vocab, layers, align;
  NxTableRouteLayer layer[NX_TABLE_LAYERS];
} NxTableRouteArgs;
int nx_moe_table_route(const NxTableRouteArgs* args, nx_stream_t stream);

// Experts by a learned router.  A row's scores are s = sigmoid(logits), its choice scores s + correction.  With n_groups > 1 the
// experts form equal groups of neighbours, a group's score is the sum of its two largest choice scores, and only experts of
// the `keep` best groups can be chosen.  The `top` largest choice scores win (ties: the lower id); weight = s / (sum of the
// chosen s + 1e-20).  The assignments are sorted as above.  With by_slot, row r of h is copied to by_slot at each of its slots.
typedef struct NxGateRouteArgs {
  const float* logits;       // [n, ld]
  const float* correction;   // [experts]
  int32_t* expert;           // [n, top]
  float* weight;             // [n, top]
  int32_t* slots;            // [n, top]
  int32_t* rows;             // [max_slots]
  int32_t* start;            // [experts]
  int32_t* count;            // [experts]
  int32_t* groups;           // [max_slots / align]
  const void* h;             // [n], rows of row_bytes (a multiple of 16)
  void* by_slot;             // [max_slots], may be null
  int64_t ld;
  int32_t n, experts, top, n_groups, keep, align, max_slots, row_bytes;   // experts <= 1024, top <= 32
} NxGateRouteArgs;
int nx_moe_gate_route(const NxGateRouteArgs* args, nx_stream_t stream);

// out[slot] = act(W[e] x[row of slot]) for every slot of every expert; `rows` null: row = slot.  act: NX_ACT_NONE or RELU2.
// gated (few rows only): the rows of W are turns of eight gates and eight values (n counts both), out has n / 2 columns.
// start and count null: every group has slots 0..m (a matrix per head).
typedef struct NxExpertGemmArgs {
  const void* x;           // [., ldx]
  const int32_t* rows;
  const void* w;           // [experts, n, ldw]
  void* out;               // [slots, ldo]
  const int32_t* start;
  const int32_t* count;
  const int32_t* groups;   // FP32 form: expert per tile of `align` slots
  int64_t ldx, ldw, stride_w, ldo;
  int32_t experts, n, k, act, tiles, align;
  int64_t group_x, group_out;  // few rows: what a group adds to the addresses of x and out (elements)
  int32_t m;                   // few rows: most slots of a group
  int32_t gated;
  NxGlu glu;
} NxExpertGemmArgs;
// few rows per expert, BF16: the weights stream through registers once per 32 rows; k, ldx, ldw, group_x multiples of 8
int nx_expert_skinny(const NxExpertGemmArgs* args, nx_stream_t stream);
// FP32, align 32
int nx_expert_f32(const NxExpertGemmArgs* args, nx_stream_t stream);

#ifdef __cplusplus
}
#endif
