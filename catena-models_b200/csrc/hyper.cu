// Hyper-connections: the residual stream as S copies of width W per token, float, [rows][S][W].  A sublayer reads a
// weighted sum of the copies and its result is written back to all of them at once:
//
//   u = sum_s a[s] x_s                         what a sublayer's norm takes   (a: S numbers of that sublayer)
//   x_t <- sum_s M[s][t] x_s + c[t] y          y = the sublayer's result      (M: S x S, from s to t; c: S numbers)
//
// One kernel does the write behind a sublayer and the read in front of the next one: the new copies, their weighted sum
// u and its layer norm n = (u - mean) / sqrt(variance + eps) * w, rounded to activations.  The same kernel opens the
// stream (all copies equal to one row) and reads it alone (a norm over copies that stay as they are; the end of the
// stack reads with a[s] = 1).  A block owns a row, a thread its own columns of all copies, so the copies may be updated
// in place; sums run in a fixed order and do not depend on the other rows of the launch.
#include "residual_terms.cuh"

#define HC_THREADS 256
#define HC_MAX_STREAMS 8

struct HyperArgs {
    float* x_out;              // [rows][S][W]: the new copies, or null: they stay as they are (read only)
    const float* x_in;         // [rows][S][W] (may be x_out), or [rows][W] when `open`
    int open;                  // 1: every copy becomes the row of x_in; M, c and the terms are not used
    const float* mix;          // [S][S] float, or null: the copies keep their values
    const float* put;          // [S] float: c
    const float* read;         // [S] float: a of whatever reads next, or null: no norm
    const float* w;            // [W] float: the layer norm's weight
    float eps;
    int W;
};

template <typename T, int VEC>
__device__ __forceinline__ void load_cols(const void* p, bool f32, long long i, float* out) {
    if constexpr (VEC == 4) {
        if (f32 || sizeof(T) == 4) {
            const float4 t = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
            out[0] = t.x; out[1] = t.y; out[2] = t.z; out[3] = t.w;
        } else {
            const uint2 raw = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p) + i);
            const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
            const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
            out[0] = a.x; out[1] = a.y; out[2] = b.x; out[3] = b.y;
        }
    } else {
        out[0] = f32 ? reinterpret_cast<const float*>(p)[i] : to_f32(reinterpret_cast<const T*>(p)[i]);
    }
}
template <int VEC>
__device__ __forceinline__ void store_floats(float* p, const float* v) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else p[0] = v[0];
}
template <typename T, int VEC>
__device__ __forceinline__ void store_act(T* p, const float* v) {
    if constexpr (VEC == 4 && sizeof(T) == 2) {
        uint2 raw;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
        h[0] = __floats2bfloat162_rn(v[0], v[1]);
        h[1] = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = raw;
    } else if constexpr (VEC == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        p[0] = from_f32<T>(v[0]);
    }
}

// the terms of row r at columns c .. c + VEC - 1, added to each other in their order (terms_at, VEC columns at a time)
template <typename T, int VEC>
__device__ __forceinline__ void terms_cols(const ResidualTerms& terms, long long r, int W, int c, float* add) {
#pragma unroll
    for (int v = 0; v < VEC; ++v) add[v] = 0.f;
    for (int i = 0; i < terms.n; ++i) {
        const ResidualTerm& t = terms.t[i];
        float s[VEC];
#pragma unroll
        for (int v = 0; v < VEC; ++v) s[v] = 0.f;
        for (int j = 0; j < t.per_row; ++j) {
            const long long piece = t.index ? t.index[r * t.per_row + j] : r * t.per_row + j;
            if (piece < 0) continue;
            float x[VEC];
            load_cols<T, VEC>(t.p, t.is_f32, piece * W + c, x);
            if (t.weights) {
                const float wt = t.weights[r * t.per_row + j];
#pragma unroll
                for (int v = 0; v < VEC; ++v) s[v] = fmaf(wt, x[v], s[v]);
            } else {
#pragma unroll
                for (int v = 0; v < VEC; ++v) s[v] += x[v];
            }
        }
#pragma unroll
        for (int v = 0; v < VEC; ++v) add[v] += t.scale * s[v];
    }
}

template <typename T, int S, int VEC>
__global__ void __launch_bounds__(HC_THREADS)
hyper_kernel(const HyperArgs a, T* __restrict__ n_out, const ResidualTerms terms) {
    extern __shared__ __align__(16) float row[];
    __shared__ float scratch[32];
    float M[S][S], put[S], rd[S];                   // constants of the model: read before the wait
#pragma unroll
    for (int t = 0; t < S; ++t) {
        put[t] = a.put ? a.put[t] : 0.f;
        rd[t] = a.read ? a.read[t] : 0.f;
#pragma unroll
        for (int s = 0; s < S; ++s) M[s][t] = a.mix ? a.mix[s * S + t] : 0.f;
    }
    pdl_trigger();
    pdl_wait();
    const int W = a.W;
    const long long r = blockIdx.x;
    float sum = 0.f;
    for (int c = threadIdx.x * VEC; c < W; c += HC_THREADS * VEC) {
        float x[S][VEC];
        if (a.open) {
            float e[VEC];
            load_cols<T, VEC>(a.x_in, true, r * W + c, e);
#pragma unroll
            for (int s = 0; s < S; ++s)
#pragma unroll
                for (int v = 0; v < VEC; ++v) x[s][v] = e[v];
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s) load_cols<T, VEC>(a.x_in, true, (r * S + s) * W + c, x[s]);
        }
        if (a.mix) {
            float y[VEC];
            terms_cols<T, VEC>(terms, r, W, c, y);
            float z[S][VEC];
#pragma unroll
            for (int t = 0; t < S; ++t)
#pragma unroll
                for (int v = 0; v < VEC; ++v) {
                    float acc = put[t] * y[v];
#pragma unroll
                    for (int s = S - 1; s >= 0; --s) acc = fmaf(M[s][t], x[s][v], acc);
                    z[t][v] = acc;
                }
#pragma unroll
            for (int t = 0; t < S; ++t)
#pragma unroll
                for (int v = 0; v < VEC; ++v) x[t][v] = z[t][v];
        }
        if (a.x_out) {
#pragma unroll
            for (int t = 0; t < S; ++t) store_floats<VEC>(a.x_out + (r * S + t) * W + c, x[t]);
        }
        if (n_out) {
            float u[VEC];
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                u[v] = 0.f;
#pragma unroll
                for (int t = 0; t < S; ++t) u[v] = fmaf(rd[t], x[t][v], u[v]);
                sum += u[v];
            }
            store_floats<VEC>(row + c, u);
        }
    }
    if (!n_out) return;
    const float mean = block_sum(sum, scratch) / (float)W;
    float ss = 0.f;
    for (int c = threadIdx.x * VEC; c < W; c += HC_THREADS * VEC)      // every thread reads back what it stored itself
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
            const float d = row[c + v] - mean;
            ss = fmaf(d, d, ss);
        }
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)W + a.eps);
    for (int c = threadIdx.x * VEC; c < W; c += HC_THREADS * VEC) {
        float n[VEC];
#pragma unroll
        for (int v = 0; v < VEC; ++v) n[v] = ((row[c + v] - mean) * inv) * a.w[c + v];
        store_act<T, VEC>(n_out + r * W + c, n);
    }
}

template <typename T>
static int launch_hyper(const HyperArgs& a, T* n_out, const ResidualTerms& terms, int rows, int S, cudaStream_t st) {
    const size_t smem = (size_t)a.W * sizeof(float);
    bool vec = a.W % 4 == 0 && (((uintptr_t)a.x_out | (uintptr_t)a.x_in) & 15) == 0 && ((uintptr_t)n_out & (4 * sizeof(T) - 1)) == 0;
    for (int i = 0; i < terms.n; ++i)
        vec = vec && ((uintptr_t)terms.t[i].p & (terms.t[i].is_f32 ? 15 : 4 * sizeof(T) - 1)) == 0;
#define HC_LAUNCH(SS, VV)                                                                                                  \
    do {                                                                                                                   \
        if (smem > 48 * 1024)                                                                                              \
            cudaFuncSetAttribute(hyper_kernel<T, SS, VV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);         \
        cm_launch(hyper_kernel<T, SS, VV>, rows, HC_THREADS, smem, st, a, n_out, terms);                                   \
    } while (0)
#define HC_CASE(SS)                    \
    case SS:                           \
        if (vec) HC_LAUNCH(SS, 4);     \
        else HC_LAUNCH(SS, 1);         \
        break;
    switch (S) {
        HC_CASE(1) HC_CASE(2) HC_CASE(3) HC_CASE(4) HC_CASE(5) HC_CASE(6) HC_CASE(7) HC_CASE(8)
        default: CM_REFUSE("hyper_connect: %d streams (1 to %d)", S, HC_MAX_STREAMS);
    }
#undef HC_CASE
#undef HC_LAUNCH
    CM_CHECK_LAUNCH();
    return CM_OK;
}

// See HyperArgs; terms as for cm_residual_add_norm.
extern "C" int cm_hyper_connect(int dt, float* x_out, const float* x_in, int open, const float* mix, const float* put,
                                const float* read, const float* w, float eps, void* n_out, int n_terms,
                                const void* const* term_ptr, const float* term_scale, const int* term_per_row,
                                const int* term_is_f32, const int* const* term_index, const float* const* term_weights,
                                int rows, int S, int W, cudaStream_t st) {
    if (rows <= 0) return CM_OK;
    if (n_terms < 0 || n_terms > R32_MAX_TERMS) CM_REFUSE("hyper_connect: %d terms (at most %d)", n_terms, R32_MAX_TERMS);
    if ((mix == nullptr) != (put == nullptr)) CM_REFUSE("hyper_connect: mix and put come together");
    if (open && mix) CM_REFUSE("hyper_connect: opening the stream mixes nothing");
    if (n_out && (!read || !w)) CM_REFUSE("hyper_connect: a norm needs its read factors and its weight");
    if ((size_t)W * sizeof(float) > 200 * 1024) CM_REFUSE("hyper_connect: a row of %d floats does not fit shared memory", W);
    ResidualTerms terms;
    fill_terms(terms, n_terms, term_ptr, term_scale, term_per_row, term_is_f32, term_index, term_weights);
    const HyperArgs a = {x_out, x_in, open, mix, put, read, w, eps, W};
    if (dt == DT_F32) return launch_hyper<float>(a, (float*)n_out, terms, rows, S, st);
    if (dt == DT_BF16) return launch_hyper<bf16>(a, (bf16*)n_out, terms, rows, S, st);
    return CM_ERR_DTYPE;
}
