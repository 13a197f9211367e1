// What a sublayer adds to a float residual stream, as the residual kernels read it (residual32.cu, hyper.cu).
#pragma once
#include "common.cuh"

#define R32_MAX_TERMS 4

// One term of a residual sum: rows of `per_row` consecutive pieces each (a routed feed-forward leaves
// one piece per chosen expert), stored as float or as activations, times a constant.
struct ResidualTerm {
    const void* p;
    const int* index;      // null: piece j of row r is row r * per_row + j; else row index[r * per_row + j] (negative: none)
    const float* weights;  // null, or a factor per piece: weights[r * per_row + j] (a routed feed-forward's weights on its experts' outputs)
    float scale;
    int per_row;           // 0: one row that is added to every row (a bias)
    int is_f32;
};
struct ResidualTerms {
    ResidualTerm t[R32_MAX_TERMS];
    int n;
};

template <typename T>
__device__ __forceinline__ float term_at(const ResidualTerm& t, long long i) {
    return t.is_f32 ? reinterpret_cast<const float*>(t.p)[i] : to_f32(reinterpret_cast<const T*>(t.p)[i]);
}

// sum_i scale_i * sum_j (weights_i[j]) term_i[row * per_row_i + j] at column c: the terms are added to each other in their order.
template <typename T>
__device__ __forceinline__ float terms_at(const ResidualTerms& terms, long long r, int H, int c) {
    float add = 0.f;
    for (int i = 0; i < terms.n; ++i) {
        const ResidualTerm& t = terms.t[i];
        float s = t.per_row ? 0.f : term_at<T>(t, c);
        for (int j = 0; j < t.per_row; ++j) {
            const long long piece = t.index ? t.index[r * t.per_row + j] : r * t.per_row + j;
            if (piece >= 0) {
                const float v = term_at<T>(t, piece * H + c);
                s = t.weights ? fmaf(t.weights[r * t.per_row + j], v, s) : s + v;
            }
        }
        add += t.scale * s;
    }
    return add;
}

static void fill_terms(ResidualTerms& terms, int n_terms, const void* const* term_ptr, const float* term_scale,
                       const int* term_per_row, const int* term_is_f32, const int* const* term_index,
                       const float* const* term_weights) {
    terms.n = n_terms;
    for (int i = 0; i < R32_MAX_TERMS; ++i) {
        terms.t[i].p = i < n_terms ? term_ptr[i] : nullptr;
        terms.t[i].index = i < n_terms ? term_index[i] : nullptr;
        terms.t[i].weights = i < n_terms ? term_weights[i] : nullptr;
        terms.t[i].scale = i < n_terms ? term_scale[i] : 0.f;
        terms.t[i].per_row = i < n_terms ? term_per_row[i] : 0;
        terms.t[i].is_f32 = i < n_terms ? term_is_f32[i] : 0;
    }
}
