// What stands between an attention layer's packed projection and its attention kernel, for layers with more between them
// than cm_qk_prepare knows: biases on q, k and v, a norm per query and key head, a rotation of neighbouring or of opposite
// channels over the leading part of a head, values mixed with another layer's values of the same token, and the cache write,
// as one pass over the rows.
//
//   row: [ q: QH * HD | k: KVH * HD | v: KVH * HD | ... ]   (row stride ld; heads padded with zero channels allowed)
//   q, k:  u = x + bias;  u <- (u / sqrt(sum u^2 / norm_dim + eps)) * w   (w given);  pairs of channels turned by position * rate
//   v:     u = x + bias;  u <- (1 - lam) u + lam v_first                  (v_first given: rows of the layer that made them)
//
// Everything between the load and the one rounding at the end is float.  q, k and v are written back in place; k and v also
// go to the cache entry of (slot, position) when a pool is given.  Rows of padding (tok_seq < 0) are left alone.
#include "common.cuh"
#include "head_prepare.h"
#include <math.h>

// One warp per token and run of passes.  A head's channels are cut into runs of eight, LPH = HD / 8 lanes own one run each,
// so a warp has 32 / LPH heads of its token in hand at a time; sine and cosine are formed once per lane and serve every head.
// PAIRED: the rotation pairs channels 2i and 2i + 1, else i and i + HD / 2 (the partner sits LPH / 2 lanes away).
template <typename T, bool PAIRED>
__global__ void __launch_bounds__(128)
head_prepare_kernel(const HeadPrepareArgs a, int passes_per_warp) {
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x;
    const long long t = blockIdx.x * (long long)blockDim.y + threadIdx.y;
    if (t >= a.rows || a.tok_seq[t] < 0) return;
    const int HD = a.HD, QH = a.QH, KVH = a.KVH, LPH = HD >> 3, HPP = 32 / LPH;
    const int sub = lane % LPH, hsel = lane / LPH;          // lanes past HPP * LPH idle along
    const int c0 = sub * 8;
    const int pos = a.tok_pos[t];
    constexpr int NA = PAIRED ? 4 : 8;
    float sn[NA], cs[NA];
#pragma unroll
    for (int e = 0; e < NA; ++e) {
        const int pair = PAIRED ? sub * 4 + e : (sub % max(1, LPH >> 1)) * 8 + e;
        sn[e] = 0.f;
        cs[e] = 1.f;
        if (pair < a.pairs) {
            sincosf((float)pos * a.rate[pair], &sn[e], &cs[e]);
            sn[e] *= a.mag;
            cs[e] *= a.mag;
        }
    }
    int page = -1, row = 0;
    if (a.pool) {
        const int b = a.tok_seq[t];
        if (a.ring == 0 || pos + a.ring >= a.seq_end[b]) {
            const int entry = a.ring ? pos % a.ring : pos;
            page = a.ptab[(long long)a.seq_slot[b] * a.ptab_stride + entry / PAGE_TOKENS];
            row = entry % PAGE_TOKENS;
        }
    }
    const float lam = a.v_first ? a.lam[0] : 0.f;
    const int n_heads = QH + 2 * KVH;
    const int pass0 = blockIdx.y * passes_per_warp;
    for (int pass = pass0; pass < pass0 + passes_per_warp; ++pass) {
        const int head = pass * HPP + hsel;
        const bool live = hsel < HPP && head < n_heads;
        const bool is_v = head >= QH + KVH;
        T* x = (T*)a.qkv + t * a.ld + (long long)head * HD + c0;
        float u[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (live) {
            load8f<T>(x, u);
            if (a.bias) {
                float bs[8];
                load8f<float>(a.bias + (long long)head * HD + c0, bs);
#pragma unroll
                for (int e = 0; e < 8; ++e) u[e] += bs[e];
            }
        }
        const float* w = head < QH ? a.wq : (is_v ? nullptr : a.wk);
        if (a.wq || a.wk) {                                 // the shuffles are for the whole warp
            float ss = 0.f, tot = 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss = fmaf(u[e], u[e], ss);
            for (int j = 0; j < LPH; ++j) tot += __shfl_sync(0xffffffffu, ss, (hsel * LPH + j) & 31);
            if (w && live) {
                const float inv = 1.f / sqrtf(tot / (float)a.norm_dim + a.eps);
                float wv[8];
                load8f<float>(w + c0, wv);
#pragma unroll
                for (int e = 0; e < 8; ++e) u[e] = (u[e] * inv) * wv[e];
            }
        }
        if (PAIRED) {
            if (!is_v) {
#pragma unroll
                for (int p = 0; p < 4; ++p) {
                    const float lo = u[2 * p], hi = u[2 * p + 1];
                    u[2 * p] = lo * cs[p] - hi * sn[p];
                    u[2 * p + 1] = hi * cs[p] + lo * sn[p];
                }
            }
        } else if (a.pairs > 0) {
            const int half = LPH >> 1;
            const bool low = sub < half;
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const float other = __shfl_sync(0xffffffffu, u[e], (low ? lane + half : lane - half) & 31);
                if (!is_v) u[e] = low ? u[e] * cs[e % NA] - other * sn[e % NA] : u[e] * cs[e % NA] + other * sn[e % NA];
            }
        }
        if (!live) continue;
        if (is_v && a.v_first) {
            const int vc = (head - QH - KVH) * a.DV + c0;   // the run's first channel, counted over the values without padding
            const T* f = (const T*)a.v_first + t * a.ld_first;
            float o[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
            if (a.vec_first) {
                if (c0 < a.DV) load8f<T>(f + (vc / a.DV1) * a.HD1 + vc % a.DV1, o);
            } else {
#pragma unroll
                for (int e = 0; e < 8; ++e) o[e] = c0 + e < a.DV ? to_f32(f[((vc + e) / a.DV1) * a.HD1 + (vc + e) % a.DV1]) : 0.f;
            }
#pragma unroll
            for (int e = 0; e < 8; ++e)
                if (c0 + e < a.DV) u[e] = fmaf(lam, o[e], (1.f - lam) * u[e]);
        }
        store8f<T>(x, u);
        if (page >= 0 && head >= QH) {
            const int plane = is_v ? 1 : 0;
            store8f<T>(kv_tile((T*)a.pool, plane, a.pages, page, head - QH - plane * KVH, KVH, HD) + (long long)row * HD + c0, u);
        }
    }
}

template <typename T>
static int launch_head_prepare(const HeadPrepareArgs& a, cudaStream_t st) {
    const int hpp = 32 / (a.HD / 8), passes = (a.QH + 2 * a.KVH + hpp - 1) / hpp;
    // a warp walks several passes of its token when the tokens alone give the SMs enough warps
    int ppw = passes;
    while (ppw > 1 && a.rows * ((passes + ppw - 1) / ppw) < 8192) ppw = (ppw + 1) / 2;
    dim3 block(32, 4), grid((unsigned)((a.rows + 3) / 4), (passes + ppw - 1) / ppw);
    if (a.interleaved) cm_launch(head_prepare_kernel<T, true>, grid, block, 0, st, a, ppw);
    else cm_launch(head_prepare_kernel<T, false>, grid, block, 0, st, a, ppw);
    CM_CHECK_LAUNCH();
    return CM_OK;
}

extern "C" int cm_head_prepare(int dt, const HeadPrepareArgs* args, cudaStream_t st) {
    HeadPrepareArgs a = *args;
    if (a.rows <= 0) return CM_OK;
    const size_t esz = dt == DT_F32 ? 4 : 2;
    if (a.HD < 16 || a.HD % 16 || a.HD > CM_MAX_HEAD_DIM) CM_REFUSE("head_prepare: head size %d (multiples of 16 up to %d)", a.HD, CM_MAX_HEAD_DIM);
    if ((a.ld * esz) % 16 || (((uintptr_t)a.qkv | (uintptr_t)a.pool | (uintptr_t)a.wq | (uintptr_t)a.wk | (uintptr_t)a.bias) & 15))
        CM_REFUSE("head_prepare: rows, constants and cache aligned to 16 bytes");
    if (a.ring % PAGE_TOKENS) CM_REFUSE("head_prepare: ring of %d entries is no multiple of %d", a.ring, PAGE_TOKENS);
    if (a.norm_dim < 1 || a.norm_dim > a.HD || a.pairs < 0 || a.pairs > a.HD / 2 || (a.pairs && !a.rate))
        CM_REFUSE("head_prepare: a norm over %d and a rotation of %d pairs in heads of %d", a.norm_dim, a.pairs, a.HD);
    if (a.v_first && (!a.lam || a.DV < 1 || a.DV > a.HD || a.DV1 < 1 || a.HD1 < a.DV1))
        CM_REFUSE("head_prepare: values of %d channels mixed with values of %d", a.DV, a.DV1);
    a.vec_first = a.v_first && a.DV % 8 == 0 && a.DV1 % 8 == 0 && a.HD1 % 8 == 0 && (a.ld_first * esz) % 16 == 0 &&
                  ((uintptr_t)a.v_first & 15) == 0;
    if (dt == DT_F32) return launch_head_prepare<float>(a, st);
    if (dt == DT_BF16) return launch_head_prepare<bf16>(a, st);
    return CM_ERR_DTYPE;
}
