// One summand of a sublayer's output as the kernels that add it into the stream take it (see Branch in host/parts.hpp):
// exactly one of
//   t          a dense tensor [T, d] in the activations' type;
//   parts      the unsummed float32 parts [n_splits][T, d] of a product whose contraction was cut;
//   y          rows of routed experts, sum_k wts[t, k] * y[pair_row[t, k], :]; a negative pair_row stands for an identity
//              expert, whose output is the sublayer's input: row t of `input` (dense [T, d], the activations' type), or with
//              input == null the stream itself;
// or none of them (all null).
#pragma once

struct ImpBranchTerm {
    const void* t;
    const float* parts;
    int n_splits;
    const void* y;
    const int* pair_row;    // [T, top]
    const float* wts;       // [T, top]
    int top;
    const void* input;
};
