// What the kernels of the gated delta rule take (delta.cu); the Python binding fills the same record (kernels._DeltaArgs).
#pragma once
#include <cuda_runtime.h>

struct DeltaArgs {
    const void* proj;             // [rows][ldp] activations: q (G D channels) | k (G D) | v (H DV) | output gate (H DV)
    long long ldp;
    const float* gates;           // [rows][ldg] float: H pre-activations of beta, then H of the decay (not for delta_step)
    long long ldg;
    const void* x;                // delta_step: the mixer's input [rows][W] activations, and the rows of both gate
    const void* w_gates;          //             projections [2 H][W] (beta's, then the decay's), same type
    int W;
    const float *rate, *dt_bias;  // [H] float: exp(A_log), and what is added to the decay's pre-activation
    const float* taps;            // [C][K] float, C = 2 G D + H DV
    const float* norm_w;          // [H * DV] float (a weight per value channel, repeated for every head)
    float* state;                 // [slots][state_stride]: S [H][D][DV], then (K > 1) a ring of K rows of C projected channels
    long long state_stride;
    void* out;                    // [rows][ldo] activations: the heads' outputs after norm and gate
    long long ldo;
    float *qk;                    // scratch [rows][2 G D]: unit q (times q_scale) | unit k
    void* v;                      // scratch [rows][H DV] activations: v behind the taps and silu
    float* lb;                    // scratch [rows][2 H]: log decay | beta
    float* raw;                   // scratch [rows][H DV]: the heads' outputs before norm and gate
    const int *tok_seq, *tok_pos, *seq_start, *seq_pos0, *seq_slot;
    long long rows;
    int B, H, G, D, DV, K;
    float q_scale, unit_eps, eps;
    int from_zero;                // every sequence of the step starts at position 0
    float* chunks;                // scratch of the chunked form, or null: the serial scan
    int max_len;                  // most rows that a sequence brings
};

// The recurrence of a step with norm and gate, in chunks (delta_chunk.cu); a.chunks is its scratch.
template <typename T>
int delta_chunked(const DeltaArgs& a, cudaStream_t st);
