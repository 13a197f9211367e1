// Row-wise kernels for models whose residual stream is kept in float whatever the activation type:
// a norm that reads float rows and writes activations, the residual sum of several terms fused with
// the norm of whatever runs next, and the concatenation [x; x0] that a looped stack feeds to the
// projection at the start of a pass.
//
// The norm is a root-mean-square norm (kind 0), a dynamic tanh (kind 1: y = tanh(alpha x) * w + b, which takes
// no statistics of the row; alpha is read from the device) or a layer norm without a shift (kind 2: y = (x - mean) /
// sqrt(variance + eps) * w, the variance being the mean of the squared distances from the mean).
//
// A row is held in shared memory between the two passes over it (sum of squares, then scaling), so the
// width is bounded by shared memory only.  All sums are float and run in a fixed order.
#include "common.cuh"
#include "residual_terms.cuh"

#define R32_THREADS 256
#define NORM_RMS 0
#define NORM_DYT 1
#define NORM_LAYER 2

// A staged row moved to mean zero (`sum`: this thread's share of the row's sum; every thread touches its own columns
// only), and the sum of the squares of what is left.
__device__ __forceinline__ float centre_row(float* row, int H, float sum, float* scratch) {
    const float mean = block_sum(sum, scratch) / (float)H;
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float d = row[c] - mean;
        row[c] = d;
        ss += d * d;
    }
    return block_sum(ss, scratch);
}

// y = T((x * inv) * w), inv = 1 / sqrt(mean(x^2) + eps) (layer norm: of the row moved to mean zero); or
// T(tanh(alpha x) * w + b); x float.
template <typename T>
__global__ void __launch_bounds__(R32_THREADS)
norm_f32in_kernel(T* __restrict__ y, const float* __restrict__ x, const float* __restrict__ w, int H, float eps,
                  int kind, const float* __restrict__ alpha, const float* __restrict__ shift) {
    extern __shared__ float row[];
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    const float* xr = x + (long long)blockIdx.x * H;
    if (kind == NORM_DYT) {
        const float al = alpha[0];
        T* yd = y + (long long)blockIdx.x * H;
        for (int c = threadIdx.x; c < H; c += R32_THREADS) yd[c] = from_f32<T>(fmaf(tanhf(al * xr[c]), w[c], shift[c]));
        return;
    }
    float ss = 0.f, sum = 0.f;
    for (int c = threadIdx.x; c < H; c += R32_THREADS) {
        const float v = xr[c];
        row[c] = v;
        ss += v * v;
        sum += v;
    }
    if (kind == NORM_LAYER) ss = centre_row(row, H, sum, scratch);
    else ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)H + eps);
    T* yr = y + (long long)blockIdx.x * H;
    for (int c = threadIdx.x; c < H; c += R32_THREADS) yr[c] = from_f32<T>((row[c] * inv) * w[c]);
}

// h += sum_i scale_i * sum_j term_i[row * per_row_i + j] (+ bias);  n = T(norm(h) * w) when n is given.
// The terms are added to each other first, in their order, and their sum to h: x + (mixer + feed-forward).
template <typename T>
__global__ void __launch_bounds__(R32_THREADS)
residual_add_norm_kernel(float* __restrict__ h, T* __restrict__ n_out, ResidualTerms terms,
                         const float* __restrict__ bias, const float* __restrict__ w, int H, float eps,
                         int kind, const float* __restrict__ alpha, const float* __restrict__ shift) {
    extern __shared__ float row[];
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    const long long r = blockIdx.x;
    float* hr = h + r * H;
    float ss = 0.f, sum = 0.f;
    for (int c = threadIdx.x; c < H; c += R32_THREADS) {
        float v = hr[c] + terms_at<T>(terms, r, H, c);
        if (bias) v += bias[c];
        hr[c] = v;
        row[c] = v;
        ss += v * v;
        sum += v;
    }
    if (!n_out) return;
    T* nr = n_out + r * H;
    if (kind == NORM_DYT) {                          // every thread reads back what it stored itself
        const float al = alpha[0];
        for (int c = threadIdx.x; c < H; c += R32_THREADS) nr[c] = from_f32<T>(fmaf(tanhf(al * row[c]), w[c], shift[c]));
        return;
    }
    if (kind == NORM_LAYER) ss = centre_row(row, H, sum, scratch);
    else ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)H + eps);
    for (int c = threadIdx.x; c < H; c += R32_THREADS) nr[c] = from_f32<T>((row[c] * inv) * w[c]);
}

// The norm behind the sum (a post-norm layer), optionally followed by an average over the depth of the stack:
//   x = norm(h_scale * h + terms) * w
//   without `hist`:  h <- x
//   with `hist` [n_hist][rows][H] (entry j at hist + j * hist_stride): entry n_hist - 1 <- x, and
//                    h <- sum over j < n_hist of coef[j] * entry j          (j ascending; the last entry is x itself)
//   n_out <- T(h) when given: the rows as the next reader's products take them.
template <typename T>
__global__ void __launch_bounds__(R32_THREADS)
postnorm_residual_kernel(float* __restrict__ h, T* __restrict__ n_out, ResidualTerms terms, float h_scale,
                         const float* __restrict__ w, int H, float eps, float* __restrict__ hist, long long hist_stride,
                         int n_hist, const float* __restrict__ coef) {
    extern __shared__ float row[];
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    const long long r = blockIdx.x;
    float* hr = h + r * H;
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += R32_THREADS) {
        const float v = fmaf(h_scale, hr[c], terms_at<T>(terms, r, H, c));
        row[c] = v;
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)H + eps);
    for (int c = threadIdx.x; c < H; c += R32_THREADS) {     // every thread reads back what it stored itself
        float x = (row[c] * inv) * w[c];
        if (hist) {
            hist[(long long)(n_hist - 1) * hist_stride + r * H + c] = x;
            float mix = 0.f;
            for (int j = 0; j + 1 < n_hist; ++j) mix = fmaf(coef[j], hist[(long long)j * hist_stride + r * H + c], mix);
            x = fmaf(coef[n_hist - 1], x, mix);
        }
        hr[c] = x;
        if (n_out) n_out[r * H + c] = from_f32<T>(x);
    }
}

// The norm on what is added: h += norm(terms) * w.  n_out <- T(h) when given, or with w_next T(norm(h) * w_next): the rows
// as the next reader takes them.
template <typename T>
__global__ void __launch_bounds__(R32_THREADS)
outnorm_residual_kernel(float* __restrict__ h, T* __restrict__ n_out, ResidualTerms terms, const float* __restrict__ w,
                        const float* __restrict__ w_next, int H, float eps, float eps_next) {
    extern __shared__ float row[];
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    const long long r = blockIdx.x;
    float* hr = h + r * H;
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += R32_THREADS) {
        const float v = terms_at<T>(terms, r, H, c);
        row[c] = v;
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)H + eps);
    float hs = 0.f;
    for (int c = threadIdx.x; c < H; c += R32_THREADS) {     // every thread reads back what it stored itself
        const float x = fmaf(row[c] * inv, w[c], hr[c]);
        hr[c] = x;
        row[c] = x;
        hs += x * x;
        if (n_out && !w_next) n_out[r * H + c] = from_f32<T>(x);
    }
    if (!n_out || !w_next) return;
    hs = block_sum(hs, scratch);
    const float inv_next = 1.f / sqrtf(hs / (float)H + eps_next);
    for (int c = threadIdx.x; c < H; c += R32_THREADS) n_out[r * H + c] = from_f32<T>((row[c] * inv_next) * w_next[c]);
}

// The same with 16-byte accesses for terms that are plain rows (one piece a row, or one row for all): a thread owns four
// consecutive columns at a time and keeps them in registers.
#define R32_VEC_MAX 8              // chunks of 4 * R32_THREADS columns: rows of up to 8,192
template <typename T>
__device__ __forceinline__ float4 term4(const ResidualTerm& t, long long i) {
    if (t.is_f32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(t.p) + i);
    const T* p = reinterpret_cast<const T*>(t.p) + i;
    return make_float4(to_f32(p[0]), to_f32(p[1]), to_f32(p[2]), to_f32(p[3]));
}
__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(bf16* p, float4 v) {
    __nv_bfloat162 h[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<uint2*>(h);
}
template <typename T, int CH>
__global__ void __launch_bounds__(R32_THREADS)
outnorm_residual_vec_kernel(float* __restrict__ h, T* __restrict__ n_out, ResidualTerms terms, const float* __restrict__ w,
                            const float* __restrict__ w_next, int H, float eps, float eps_next) {
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    const long long r = blockIdx.x;
    float* hr = h + r * H;
    float4 y[CH], x[CH];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < CH; ++k) {
        const int c = (k * R32_THREADS + threadIdx.x) * 4;
        y[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c >= H) continue;
        x[k] = *reinterpret_cast<const float4*>(hr + c);
        for (int i = 0; i < terms.n; ++i) {
            const ResidualTerm& t = terms.t[i];
            const float4 v = term4<T>(t, (t.per_row ? r * H : 0) + c);
            y[k].x += t.scale * v.x; y[k].y += t.scale * v.y; y[k].z += t.scale * v.z; y[k].w += t.scale * v.w;
        }
        ss += y[k].x * y[k].x + y[k].y * y[k].y + y[k].z * y[k].z + y[k].w * y[k].w;
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)H + eps);
    float hs = 0.f;
#pragma unroll
    for (int k = 0; k < CH; ++k) {
        const int c = (k * R32_THREADS + threadIdx.x) * 4;
        if (c >= H) continue;
        const float4 wv = *reinterpret_cast<const float4*>(w + c);
        x[k].x = fmaf(y[k].x * inv, wv.x, x[k].x); x[k].y = fmaf(y[k].y * inv, wv.y, x[k].y);
        x[k].z = fmaf(y[k].z * inv, wv.z, x[k].z); x[k].w = fmaf(y[k].w * inv, wv.w, x[k].w);
        put4(hr + c, x[k]);
        hs += x[k].x * x[k].x + x[k].y * x[k].y + x[k].z * x[k].z + x[k].w * x[k].w;
        if (n_out && !w_next) put4(n_out + r * H + c, x[k]);
    }
    if (!n_out || !w_next) return;
    hs = block_sum(hs, scratch);
    const float inv_next = 1.f / sqrtf(hs / (float)H + eps_next);
#pragma unroll
    for (int k = 0; k < CH; ++k) {
        const int c = (k * R32_THREADS + threadIdx.x) * 4;
        if (c >= H) continue;
        const float4 wv = *reinterpret_cast<const float4*>(w_next + c);
        put4(n_out + r * H + c, make_float4((x[k].x * inv_next) * wv.x, (x[k].y * inv_next) * wv.y, (x[k].z * inv_next) * wv.z,
                                            (x[k].w * inv_next) * wv.w));
    }
}

// out[r] = T([a[r]; b[r]]) for float rows a and b of width H: the input of a projection over both.
template <typename T>
__global__ void concat_cast_kernel(T* __restrict__ out, const float* __restrict__ a, const float* __restrict__ b,
                                   long long rows, int H) {
    pdl_trigger();
    pdl_wait();
    const long long total = rows * 2 * H;
    for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long r = i / (2 * H);
        const int c = (int)(i - r * 2 * H);
        out[i] = from_f32<T>(c < H ? a[r * H + c] : b[r * H + c - H]);
    }
}

static int row_smem(int H, size_t* out) {
    *out = (size_t)H * sizeof(float);
    if (*out > 200 * 1024) CM_REFUSE("a row of %d floats does not fit shared memory", H);
    return CM_OK;
}

extern "C" int cm_norm_f32in(int dt, void* y, const float* x, const float* w, int rows, int H, float eps,
                             int kind, const float* alpha, const float* shift, cudaStream_t st) {
    if (rows <= 0) return CM_OK;
    if (kind == NORM_DYT && (!alpha || !shift)) CM_REFUSE("norm_f32in: a dynamic tanh needs its alpha and its shift");
    size_t smem;
    if (row_smem(H, &smem) != CM_OK) return CM_ERR_SHAPE;
    if (dt == DT_F32) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(norm_f32in_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        cm_launch(norm_f32in_kernel<float>, rows, R32_THREADS, smem, st, (float*)y, x, w, H, eps, kind, alpha, shift);
    } else if (dt == DT_BF16) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(norm_f32in_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        cm_launch(norm_f32in_kernel<bf16>, rows, R32_THREADS, smem, st, (bf16*)y, x, w, H, eps, kind, alpha, shift);
    } else
        return CM_ERR_DTYPE;
    CM_CHECK_LAUNCH();
    return CM_OK;
}

// terms: n_terms entries of (pointer, scale, pieces per row, stored as float?, index of the pieces or null, a weight per
// piece or null) in parallel arrays.
extern "C" int cm_residual_add_norm(int dt, float* h, void* n_out, int n_terms, const void* const* term_ptr,
                                    const float* term_scale, const int* term_per_row, const int* term_is_f32,
                                    const int* const* term_index, const float* const* term_weights, const float* bias,
                                    const float* w, int rows, int H, float eps, int kind, const float* alpha,
                                    const float* shift, cudaStream_t st) {
    if (rows <= 0) return CM_OK;
    if (n_terms < 0 || n_terms > R32_MAX_TERMS) CM_REFUSE("residual_add_norm: %d terms (at most %d)", n_terms, R32_MAX_TERMS);
    if (n_out && !w) CM_REFUSE("residual_add_norm: a norm needs its weight");
    if (n_out && kind == NORM_DYT && (!alpha || !shift)) CM_REFUSE("residual_add_norm: a dynamic tanh needs its alpha and its shift");
    size_t smem;
    if (row_smem(H, &smem) != CM_OK) return CM_ERR_SHAPE;
    ResidualTerms terms;
    fill_terms(terms, n_terms, term_ptr, term_scale, term_per_row, term_is_f32, term_index, term_weights);
    if (dt == DT_F32) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(residual_add_norm_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        cm_launch(residual_add_norm_kernel<float>, rows, R32_THREADS, smem, st, h, (float*)n_out, terms, bias, w, H, eps, kind, alpha, shift);
    } else if (dt == DT_BF16) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(residual_add_norm_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        cm_launch(residual_add_norm_kernel<bf16>, rows, R32_THREADS, smem, st, h, (bf16*)n_out, terms, bias, w, H, eps, kind, alpha, shift);
    } else
        return CM_ERR_DTYPE;
    CM_CHECK_LAUNCH();
    return CM_OK;
}

// The post-norm sum (postnorm_residual_kernel); terms as for cm_residual_add_norm.  coef: n_hist floats on the device.
extern "C" int cm_postnorm_residual(int dt, float* h, void* n_out, int n_terms, const void* const* term_ptr,
                                    const float* term_scale, const int* term_per_row, const int* term_is_f32,
                                    const int* const* term_index, const float* const* term_weights, float h_scale,
                                    const float* w, int rows, int H, float eps, float* hist, long long hist_stride,
                                    int n_hist, const float* coef, cudaStream_t st) {
    if (rows <= 0) return CM_OK;
    if (n_terms < 0 || n_terms > R32_MAX_TERMS) CM_REFUSE("postnorm_residual: %d terms (at most %d)", n_terms, R32_MAX_TERMS);
    if (!w) CM_REFUSE("postnorm_residual: the norm needs its weight");
    if (hist && (n_hist < 1 || !coef)) CM_REFUSE("postnorm_residual: an average over %d entries needs its coefficients", n_hist);
    size_t smem;
    if (row_smem(H, &smem) != CM_OK) return CM_ERR_SHAPE;
    ResidualTerms terms;
    fill_terms(terms, n_terms, term_ptr, term_scale, term_per_row, term_is_f32, term_index, term_weights);
    if (dt == DT_F32) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(postnorm_residual_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        cm_launch(postnorm_residual_kernel<float>, rows, R32_THREADS, smem, st, h, (float*)n_out, terms, h_scale, w, H, eps, hist,
                  hist_stride, n_hist, coef);
    } else if (dt == DT_BF16) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(postnorm_residual_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        cm_launch(postnorm_residual_kernel<bf16>, rows, R32_THREADS, smem, st, h, (bf16*)n_out, terms, h_scale, w, H, eps, hist,
                  hist_stride, n_hist, coef);
    } else
        return CM_ERR_DTYPE;
    CM_CHECK_LAUNCH();
    return CM_OK;
}

// The sum with the norm on what is added (outnorm_residual_kernel); terms as for cm_residual_add_norm.
template <typename T>
static int launch_outnorm(float* h, void* n_out, const ResidualTerms& terms, const float* w, const float* w_next, int rows, int H,
                          float eps, float eps_next, size_t smem, cudaStream_t st) {
    bool vec = H % 4 == 0 && H <= 4 * R32_THREADS * R32_VEC_MAX &&
               (((uintptr_t)h | (uintptr_t)w | (uintptr_t)w_next) & 15) == 0 && ((uintptr_t)n_out & (4 * sizeof(T) - 1)) == 0;
    for (int i = 0; i < terms.n; ++i)
        vec = vec && terms.t[i].per_row <= 1 && !terms.t[i].index && !terms.t[i].weights && ((uintptr_t)terms.t[i].p & 15) == 0;
    if (vec) {
        const int ch = (H + 4 * R32_THREADS - 1) / (4 * R32_THREADS);
#define ON_CASE(C) cm_launch(outnorm_residual_vec_kernel<T, C>, rows, R32_THREADS, 0, st, h, (T*)n_out, terms, w, w_next, H, eps, eps_next)
        if (ch <= 1) ON_CASE(1); else if (ch <= 2) ON_CASE(2); else if (ch <= 4) ON_CASE(4); else ON_CASE(8);
#undef ON_CASE
    } else {
        if (smem > 48 * 1024) cudaFuncSetAttribute(outnorm_residual_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        cm_launch(outnorm_residual_kernel<T>, rows, R32_THREADS, smem, st, h, (T*)n_out, terms, w, w_next, H, eps, eps_next);
    }
    CM_CHECK_LAUNCH();
    return CM_OK;
}

extern "C" int cm_outnorm_residual(int dt, float* h, void* n_out, int n_terms, const void* const* term_ptr,
                                   const float* term_scale, const int* term_per_row, const int* term_is_f32,
                                   const int* const* term_index, const float* const* term_weights, const float* w,
                                   const float* w_next, int rows, int H, float eps, float eps_next, cudaStream_t st) {
    if (rows <= 0) return CM_OK;
    if (n_terms < 1 || n_terms > R32_MAX_TERMS) CM_REFUSE("outnorm_residual: %d terms (1 to %d)", n_terms, R32_MAX_TERMS);
    if (!w || (w_next && !n_out)) CM_REFUSE("outnorm_residual: a norm needs its weight, and the next reader's norm a place for its rows");
    size_t smem;
    if (row_smem(H, &smem) != CM_OK) return CM_ERR_SHAPE;
    ResidualTerms terms;
    fill_terms(terms, n_terms, term_ptr, term_scale, term_per_row, term_is_f32, term_index, term_weights);
    if (dt == DT_F32) return launch_outnorm<float>(h, n_out, terms, w, w_next, rows, H, eps, eps_next, smem, st);
    if (dt == DT_BF16) return launch_outnorm<bf16>(h, n_out, terms, w, w_next, rows, H, eps, eps_next, smem, st);
    return CM_ERR_DTYPE;
}

extern "C" int cm_concat_cast(int dt, void* out, const float* a, const float* b, long long rows, int H, cudaStream_t st) {
    if (rows <= 0) return CM_OK;
    const long long total = rows * 2 * H;
    const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
    if (dt == DT_F32)
        cm_launch(concat_cast_kernel<float>, blocks, 256, 0, st, (float*)out, a, b, rows, H);
    else if (dt == DT_BF16)
        cm_launch(concat_cast_kernel<bf16>, blocks, 256, 0, st, (bf16*)out, a, b, rows, H);
    else
        return CM_ERR_DTYPE;
    CM_CHECK_LAUNCH();
    return CM_OK;
}
