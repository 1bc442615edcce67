// Routed feed-forward: which experts a row takes and the order in which rows are handed to them.
#pragma once
#include "linear_bf16.cuh"

namespace sk {

// Rows sorted by expert. A slot is one (row, choice) pair; sorted positions run over the experts in order, inside an expert
// in slot order, so the layout does not depend on timing.
struct RouteBuffers {
    int32_t* slot_expert = nullptr;      // [rows * top]
    float* slot_weight = nullptr;
    int32_t* slot_pos = nullptr;         // [rows * top] sorted position of a slot
    int32_t* sorted_row = nullptr;       // [rows * top] activation row of a sorted position
    float* sorted_weight = nullptr;
    RowSegment* segs = nullptr;          // runs of at most seg_rows sorted positions of one expert
    int32_t* n_segs = nullptr;
};
constexpr int ROUTE_MAX_EXPERTS = 4096;
inline int route_max_segs(int slots, int experts, int seg_rows) { return (slots < experts ? slots : experts) + slots / seg_rows; }

// z: router logits [rows][experts]. Scores are sigmoid(z); the `top` largest are taken (lowest index on ties) with their
// scores as weights, not renormalised.
int32_t launch_route(const float* z, int rows, int experts, int top, int seg_rows, const RouteBuffers& b, cudaStream_t s);

}  // namespace sk
