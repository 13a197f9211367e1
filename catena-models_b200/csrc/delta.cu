// Gated delta rule: a mixer whose heads keep a matrix S [D][DV] that is corrected towards each new key/value pair.
//
//   q, k, v    projections behind a short causal filter per channel (K taps, the last one the present row's) and silu;
//              H value heads, G heads of q and k (head h reads q/k head h / (H / G)); q and k are then unit vectors,
//              x / sqrt(sum x^2 + unit_eps), and q is multiplied by q_scale
//   decay      log g = -rate * softplus(z_a + dt_bias), one per head and token;  beta = sigmoid(z_b)
//   per head   S <- g S ;  u = beta (v - S^T k) ;  S <- S + k u^T ;  o = S^T q        (o sees the present pair)
//   output     o / rms(o) * norm weight * silu(gate)
//
// The state, and everything that enters the recurrence behind the projections and the filter, is float whatever the
// activation type.  S lives in per-slot rows of a float array, with the filter's last projected rows behind it as a
// ring (the row of position s in row s % K; a single token writes a row that nobody reads, so the ring moves on in the
// same launch).  Rows that belong to no sequence (padding) are never touched.
//
// Steps of one token per sequence run delta_step_kernel: everything from the filter to the gated output of a head in one
// block.  Longer steps run delta_prepare_kernel (filter, silu, unit vectors, gates: all rows side by side), then the
// recurrence: row by row (delta_scan_kernel) with norm and gate behind it (cm_scan_norm_gate), or, for long steps, in
// chunks of rows (delta_chunk.cu).
#include "common.cuh"
#include "delta.h"
#include "recurrent.h"
#include <math.h>

__device__ __forceinline__ float silu_f32(float x) { return x * sigmoid_f32(x); }
__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float log_decay_of(const DeltaArgs& a, int h, float z) { return -a.rate[h] * softplus_f32(z + a.dt_bias[h]); }

__host__ __device__ __forceinline__ int delta_channels(const DeltaArgs& a) { return 2 * a.G * a.D + a.H * a.DV; }
__device__ __forceinline__ float* delta_state(const DeltaArgs& a, int slot) { return a.state + (long long)slot * a.state_stride; }
__device__ __forceinline__ float* delta_ring(const DeltaArgs& a, int slot) { return delta_state(a, slot) + (long long)a.H * a.D * a.DV; }

// What the filter of channel c reads at position s <= pos of the token in row t (p0: its sequence's first position of
// the step).
template <typename T>
__device__ __forceinline__ float delta_tap(const DeltaArgs& a, int C, const float* ring, int c, long long t, int pos, int p0, int s) {
    if (s >= p0) return to_f32(((const T*)a.proj)[(t - (pos - s)) * a.ldp + c]);
    return s >= 0 ? ring[(long long)(s % a.K) * C + c] : 0.f;
}

// ------------------------------------------------------------------------------ filter, unit vectors, gates
#define DP_TOKENS 8          // rows that a warp takes one after the other
#define DP_WARPS 4

// Two neighbouring channels as floats (`pair`: as one access).
__device__ __forceinline__ float2 two_of(const bf16* p, bool pair, bool second) {
    if (pair) return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    return make_float2(to_f32(p[0]), second ? to_f32(p[1]) : 0.f);
}
__device__ __forceinline__ float2 two_of(const float* p, bool pair, bool second) {
    if (pair) return *reinterpret_cast<const float2*>(p);
    return make_float2(p[0], second ? p[1] : 0.f);
}

// A warp takes one unit of a row: a head of q, a head of k, or a run of up to 64 NP channels of v; lane l owns the channels
// 2 l, 2 l + 1 of every 64.  Units [0, G): q heads; [G, 2 G): k heads; then the runs of v; the last unit is the gates.
// Where the warp's rows all belong to one sequence, and every tap of all of them lies in the step (the usual case of a long
// prompt), the rows' inputs are fetched once, side by side, and the taps of a channel stay in registers (KF > 0: K = KF taps;
// 0: the general form alone).
template <typename T, int NP, int KF>
__global__ void __launch_bounds__(32 * DP_WARPS)
delta_prepare_kernel(const DeltaArgs a, int v_units, int pairs_ok) {
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int unit = blockIdx.y, G = a.G, D = a.D, K = a.K;
    const long long t_first = ((long long)blockIdx.x * DP_WARPS + warp) * DP_TOKENS;
    if (unit == 2 * G + v_units) {                     // the gates: a lane per (row, head)
        for (int e = lane; e < DP_TOKENS * a.H; e += 32) {
            const long long t = t_first + e / a.H;
            const int h = e % a.H;
            if (t >= a.rows || a.tok_seq[t] < 0) continue;
            a.lb[t * 2 * a.H + h] = log_decay_of(a, h, a.gates[t * a.ldg + a.H + h]);
            a.lb[t * 2 * a.H + a.H + h] = sigmoid_f32(a.gates[t * a.ldg + h]);
        }
        return;
    }
    const int C = delta_channels(a);
    const bool is_v = unit >= 2 * G;
    const int c0 = is_v ? 2 * G * D + (unit - 2 * G) * 64 * NP : unit * D;       // first channel of the unit
    const int n = is_v ? min(64 * NP, C - c0) : D;
    if constexpr (KF > 0) {
        const long long t_last = t_first + DP_TOKENS - 1;
        int b = -1;
        bool fast = pairs_ok && t_last < a.rows;
        if (fast) {
            b = a.tok_seq[t_first];
            fast = b >= 0 && a.tok_seq[t_last] == b && a.tok_pos[t_first] - (KF - 1) >= a.seq_pos0[b];
        }
        if (fast) {
            const int last = a.seq_pos0[b] + a.seq_start[b + 1] - a.seq_start[b] - (KF - 1), pos = a.tok_pos[t_first];
            float* ring = KF > 1 ? delta_ring(a, a.seq_slot[b]) : nullptr;
            float y[DP_TOKENS][NP][2], ss[DP_TOKENS];
#pragma unroll
            for (int i = 0; i < DP_TOKENS; ++i) ss[i] = 0.f;
#pragma unroll
            for (int p = 0; p < NP; ++p) {
                const int c = 64 * p + 2 * lane;
                if (c >= n) continue;                          // n is even here
                float2 u[DP_TOKENS + KF - 1];
                const T* src = (const T*)a.proj + (t_first - (KF - 1)) * a.ldp + c0 + c;
#pragma unroll
                for (int r = 0; r < DP_TOKENS + KF - 1; ++r) u[r] = two_of(src + (long long)r * a.ldp, true, true);
                float w0[KF], w1[KF];
#pragma unroll
                for (int j = 0; j < KF; ++j) {
                    w0[j] = a.taps[(long long)(c0 + c) * KF + j];
                    w1[j] = a.taps[(long long)(c0 + c + 1) * KF + j];
                }
#pragma unroll
                for (int i = 0; i < DP_TOKENS; ++i) {
                    float y0 = 0.f, y1 = 0.f;
#pragma unroll
                    for (int j = 0; j < KF; ++j) {
                        y0 = fmaf(w0[j], u[i + j].x, y0);
                        y1 = fmaf(w1[j], u[i + j].y, y1);
                    }
                    if (KF > 1 && a.from_zero && pos + i >= last)
                        *reinterpret_cast<float2*>(ring + (long long)((pos + i) % KF) * C + c0 + c) = u[i + KF - 1];
                    y[i][p][0] = silu_f32(y0);
                    y[i][p][1] = silu_f32(y1);
                    ss[i] = fmaf(y[i][p][0], y[i][p][0], fmaf(y[i][p][1], y[i][p][1], ss[i]));
                }
            }
            if (!is_v) {
#pragma unroll
                for (int i = 0; i < DP_TOKENS; ++i) ss[i] = (unit < G ? a.q_scale : 1.f) / sqrtf(warp_sum(ss[i]) + a.unit_eps);
            }
#pragma unroll
            for (int p = 0; p < NP; ++p) {
                const int c = 64 * p + 2 * lane;
                if (c >= n) continue;
#pragma unroll
                for (int i = 0; i < DP_TOKENS; ++i) {
                    const long long t = t_first + i;
                    if (is_v) {
                        T* dst = (T*)a.v + t * (long long)a.H * a.DV + (c0 - 2 * G * D) + c;
                        if constexpr (sizeof(T) == 2)
                            *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(y[i][p][0], y[i][p][1]);
                        else
                            *reinterpret_cast<float2*>(dst) = make_float2(y[i][p][0], y[i][p][1]);
                    } else {
                        *reinterpret_cast<float2*>(a.qk + t * 2 * G * D + c0 + c) = make_float2(y[i][p][0] * ss[i], y[i][p][1] * ss[i]);
                    }
                }
            }
            return;
        }
    }
    for (int i = 0; i < DP_TOKENS; ++i) {
        const long long t = t_first + i;
        if (t >= a.rows) return;
        const int b = a.tok_seq[t];
        if (b < 0) continue;
        const int pos = a.tok_pos[t], p0 = a.seq_pos0[b], slot = a.seq_slot[b];
        const T* src = (const T*)a.proj + t * a.ldp + c0;
        float y[NP][2];
        float ss = 0.f;
        const bool inside = pos - (K - 1) >= p0;       // every tap reads a row of this step
        float* ring = K > 1 ? delta_ring(a, slot) : nullptr;
        // the ring after the step: the projected rows of the sequence's last K - 1 positions (here when nothing reads it)
        const bool keep = K > 1 && a.from_zero && pos >= p0 + a.seq_start[b + 1] - a.seq_start[b] - (K - 1);
#pragma unroll
        for (int p = 0; p < NP; ++p) {
            const int c = 64 * p + 2 * lane;
            y[p][0] = y[p][1] = 0.f;
            if (c >= n) continue;
            const bool second = c + 1 < n;
            const float* w = a.taps + (long long)(c0 + c) * K;
            float2 now = make_float2(0.f, 0.f);
            if (inside) {
                for (int j = 0; j < K; ++j) {
                    now = two_of(src + c - (long long)(K - 1 - j) * a.ldp, pairs_ok, second);
                    y[p][0] = fmaf(w[j], now.x, y[p][0]);
                    if (second) y[p][1] = fmaf(w[K + j], now.y, y[p][1]);
                }
            } else {
                for (int j = 0; j < K; ++j) {
                    const int s = pos - K + 1 + j;
                    now.x = delta_tap<T>(a, C, ring, c0 + c, t, pos, p0, s);
                    y[p][0] = fmaf(w[j], now.x, y[p][0]);
                    if (second) {
                        now.y = delta_tap<T>(a, C, ring, c0 + c + 1, t, pos, p0, s);
                        y[p][1] = fmaf(w[K + j], now.y, y[p][1]);
                    }
                }
            }
            if (keep) {
                ring[(long long)(pos % K) * C + c0 + c] = now.x;
                if (second) ring[(long long)(pos % K) * C + c0 + c + 1] = now.y;
            }
            y[p][0] = silu_f32(y[p][0]);
            y[p][1] = second ? silu_f32(y[p][1]) : 0.f;
            ss = fmaf(y[p][0], y[p][0], fmaf(y[p][1], y[p][1], ss));
        }
        if (is_v) {
            T* dst = (T*)a.v + t * (long long)a.H * a.DV + (c0 - 2 * G * D);
#pragma unroll
            for (int p = 0; p < NP; ++p) {
                const int c = 64 * p + 2 * lane;
                if (c < n) dst[c] = from_f32<T>(y[p][0]);
                if (c + 1 < n) dst[c + 1] = from_f32<T>(y[p][1]);
            }
        } else {
            const float f = (unit < G ? a.q_scale : 1.f) / sqrtf(warp_sum(ss) + a.unit_eps);
            float* dst = a.qk + t * 2 * G * D + c0;
#pragma unroll
            for (int p = 0; p < NP; ++p) {
                const int c = 64 * p + 2 * lane;
                if (c < n) dst[c] = y[p][0] * f;
                if (c + 1 < n) dst[c + 1] = y[p][1] * f;
            }
        }
    }
}

// The ring after a step of several tokens on top of held ones, behind the filter: such a step overwrites rows that its
// first tokens read.
template <typename T>
__global__ void delta_ring_kernel(const DeltaArgs a) {
    pdl_trigger();
    pdl_wait();
    const int b = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x, C = delta_channels(a), K = a.K;
    const int s0 = a.seq_start[b], n = a.seq_start[b + 1] - s0;
    if (c >= C || n <= 0) return;
    const int p0 = a.seq_pos0[b], end = p0 + n;
    float* ring = delta_ring(a, a.seq_slot[b]);
    for (int s = max(p0, end - (K - 1)); s < end; ++s)
        ring[(long long)(s % K) * C + c] = to_f32(((const T*)a.proj)[(long long)(s0 + s - p0) * a.ldp + c]);
}

// ------------------------------------------------------------------------------ the recurrence, row by row
#define DS_THREADS 128
#define DS_MAX_ROWS 32            // rows of the step that a block stages at a time

// A block owns 128 / KS columns of one head's S for one sequence and walks the sequence's rows of the step in order.  A
// column's D key channels are dealt to KS neighbouring lanes in runs of four: lane ks holds the channels 4 (ks + KS x) + y,
// x < RPT / 4, y < 4, in registers.  Per row: the lanes' shares of S^T k are added by xor shuffles (the only exchange, and
// the only thing the next row waits for besides the update), u follows, S takes k u^T, and every lane leaves its share of
// the output in shared memory; once the rows of a group are through, the shares are added in lane order.
template <typename T, int RPT>
__global__ void __launch_bounds__(DS_THREADS)
delta_scan_kernel(const DeltaArgs a, int KS, int TB) {
    extern __shared__ __align__(16) float sm[];
    pdl_wait();
    const int hd = blockIdx.x, cb = blockIdx.y, b = blockIdx.z;
    const int s0 = a.seq_start[b], s1 = a.seq_start[b + 1];
    if (s1 <= s0) return;
    const int D = a.D, DV = a.DV, H = a.H, G = a.G, kh = hd / (H / G);
    const int Dp = KS * RPT;                          // a staged row's pitch, D <= Dp
    const int cols = DS_THREADS / KS;
    const int ks = threadIdx.x % KS, c = threadIdx.x / KS, j = cb * cols + c;
    const bool active = j < DV;
    float* sq = sm;                                   // [TB][Dp]
    float* sk = sq + (size_t)TB * Dp;                 // [TB][Dp]
    float* sv = sk + (size_t)TB * Dp;                 // [TB][cols]
    float* sg = sv + (size_t)TB * cols;               // [TB][2]: decay, beta
    float* part = sg + (size_t)TB * 2;                // [TB][KS][cols]
    float* st = delta_state(a, a.seq_slot[b]) + (long long)hd * D * DV;
    float S[RPT];
#pragma unroll
    for (int it = 0; it < RPT; ++it) {
        const int i = 4 * (ks + KS * (it >> 2)) + (it & 3);
        S[it] = active && i < D ? st[(long long)i * DV + j] : 0.f;
    }
    const long long ldqk = 2LL * G * D, ldv = (long long)H * DV;
    const float* Q = a.qk + (long long)kh * D;
    const float* Kp = Q + (long long)G * D;
    const T* V = (const T*)a.v + (long long)hd * DV + (long long)cb * cols;
    float* R = a.raw + (long long)hd * DV + (long long)cb * cols;
    const int n_cols = max(0, min(cols, DV - cb * cols));
    const bool vec4 = D % 4 == 0 && (((uintptr_t)a.qk) & 15) == 0;
    for (int e = threadIdx.x; e < TB * (Dp - D); e += DS_THREADS) {       // channels past D are read as zeros
        const int tt = e / (Dp - D), i = D + e - tt * (Dp - D);
        sq[(size_t)tt * Dp + i] = 0.f;
        sk[(size_t)tt * Dp + i] = 0.f;
    }
    for (long long t0 = s0; t0 < s1; t0 += TB) {
        const int nt = (int)min((long long)TB, s1 - t0);
        __syncthreads();                 // the group before is no longer read
        if (vec4) {
            const int D4 = D >> 2;
            for (int e = threadIdx.x; e < nt * D4; e += DS_THREADS) {
                const int tt = e / D4, i = (e - tt * D4) * 4;
                *reinterpret_cast<float4*>(sq + (size_t)tt * Dp + i) = *reinterpret_cast<const float4*>(Q + (t0 + tt) * ldqk + i);
                *reinterpret_cast<float4*>(sk + (size_t)tt * Dp + i) = *reinterpret_cast<const float4*>(Kp + (t0 + tt) * ldqk + i);
            }
        } else {
            for (int e = threadIdx.x; e < nt * D; e += DS_THREADS) {
                const int tt = e / D, i = e - tt * D;
                sq[(size_t)tt * Dp + i] = Q[(t0 + tt) * ldqk + i];
                sk[(size_t)tt * Dp + i] = Kp[(t0 + tt) * ldqk + i];
            }
        }
        for (int e = threadIdx.x; e < nt * cols; e += DS_THREADS) {
            const int tt = e / cols, cc = e - tt * cols;
            sv[e] = cc < n_cols ? to_f32(V[(t0 + tt) * ldv + cc]) : 0.f;
        }
        for (int tt = threadIdx.x; tt < nt; tt += DS_THREADS) {
            sg[2 * tt] = expf(a.lb[(t0 + tt) * 2 * H + hd]);
            sg[2 * tt + 1] = a.lb[(t0 + tt) * 2 * H + H + hd];
        }
        __syncthreads();
        // the operands of a row are fetched a row ahead (the shares stored below could alias them for all the compiler knows)
        float kn[RPT], qn[RPT], gn, bn, vn;
        auto fetch = [&](int tt) {
#pragma unroll
            for (int x = 0; x < RPT / 4; ++x) {
                const float4 kq = *reinterpret_cast<const float4*>(sk + tt * Dp + 4 * (ks + KS * x));
                const float4 qq = *reinterpret_cast<const float4*>(sq + tt * Dp + 4 * (ks + KS * x));
                kn[4 * x] = kq.x; kn[4 * x + 1] = kq.y; kn[4 * x + 2] = kq.z; kn[4 * x + 3] = kq.w;
                qn[4 * x] = qq.x; qn[4 * x + 1] = qq.y; qn[4 * x + 2] = qq.z; qn[4 * x + 3] = qq.w;
            }
            gn = sg[2 * tt];
            bn = sg[2 * tt + 1];
            vn = sv[tt * cols + c];
        };
        fetch(0);
        for (int tt = 0; tt < nt; ++tt) {
            float q[RPT], k[RPT];
#pragma unroll
            for (int it = 0; it < RPT; ++it) {
                k[it] = kn[it];
                q[it] = qn[it];
            }
            const float g = gn, beta = bn, vj = vn;
            fetch(min(tt + 1, nt - 1));
            float d4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int it = 0; it < RPT; ++it) {
                S[it] *= g;
                d4[it & 3] = fmaf(S[it], k[it], d4[it & 3]);
            }
            float dot = (d4[0] + d4[1]) + (d4[2] + d4[3]);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
                if (o < KS) dot += __shfl_xor_sync(0xffffffffu, dot, o);
            const float u = beta * (vj - dot);
            float a4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int it = 0; it < RPT; ++it) {
                S[it] = fmaf(k[it], u, S[it]);
                a4[it & 3] = fmaf(S[it], q[it], a4[it & 3]);
            }
            part[(tt * KS + ks) * cols + c] = (a4[0] + a4[1]) + (a4[2] + a4[3]);
        }
        __syncthreads();
        for (int e = threadIdx.x; e < nt * cols; e += DS_THREADS) {
            const int tt = e / cols, cc = e - tt * cols;
            if (cc >= n_cols) continue;
            float o = 0.f;
            for (int x = 0; x < KS; ++x) o += part[((size_t)tt * KS + x) * cols + cc];
            R[(t0 + tt) * ldv + cc] = o;
        }
    }
    pdl_trigger();
#pragma unroll
    for (int it = 0; it < RPT; ++it) {
        const int i = 4 * (ks + KS * (it >> 2)) + (it & 3);
        if (active && i < D) st[(long long)i * DV + j] = S[it];
    }
}

template <typename T>
static int launch_delta_scan(const DeltaArgs& a, cudaStream_t st) {
    // Channels per lane (a power of two from 4 to 32) and lanes per column (a power of two up to 32): as many channels as
    // leave the grid with a block or two per SM; the walk is bound by its latency per row, so what counts is how many SMs walk.
    auto lanes_for = [&](int r) { int k = 1; while (k * r < a.D) k *= 2; return k; };
    auto blocks = [&](int k) { const int cols = DS_THREADS / k; return (long long)a.H * ((a.DV + cols - 1) / cols) * a.B; };
    int rpt = 32;
    while (rpt > 4 && lanes_for(rpt / 2) <= 32 && blocks(lanes_for(rpt)) < 256) rpt /= 2;
    const int ks = lanes_for(rpt);
    if (ks > 32) CM_REFUSE("delta_scan: heads of %d key channels (up to 1024)", a.D);
    const int cols = DS_THREADS / ks, row_floats = 2 * ks * rpt + cols + 2 + DS_THREADS;
    int tb = 12288 / row_floats;                          // about 48 KB of staged rows
    tb = tb < 1 ? 1 : (tb > DS_MAX_ROWS ? DS_MAX_ROWS : tb);
    const size_t smem = (size_t)tb * row_floats * sizeof(float);
    dim3 grid(a.H, (a.DV + cols - 1) / cols, a.B);
    // In plain stream order: blocks that start early land on whichever SMs have room while the kernel before drains, several
    // on one, and stay there for the whole walk (measured on B200, 2,048 rows, 16 heads of 64 x 128: 865 against 575 us).
#define DS_LAUNCH(R) cm_launch_cluster(delta_scan_kernel<T, R>, grid, DS_THREADS, smem, st, 1, false, a, ks, tb)
    if (rpt == 4) DS_LAUNCH(4);
    else if (rpt == 8) DS_LAUNCH(8);
    else if (rpt == 16) DS_LAUNCH(16);
    else DS_LAUNCH(32);
#undef DS_LAUNCH
    CM_CHECK_LAUNCH();
    return CM_OK;
}

static int delta_check(const DeltaArgs& a) {
    if (a.D < 1 || a.D > 1024 || a.DV < 1 || a.G < 1 || a.H % a.G) CM_REFUSE("delta rule: %d heads over %d, head sizes %d x %d (keys up to 1024)", a.H, a.G, a.D, a.DV);
    if (a.K < 1 || a.K > CM_MAX_CONV_TAPS) CM_REFUSE("delta rule: %d taps (1 to %d)", a.K, CM_MAX_CONV_TAPS);
    return CM_OK;
}

template <typename T>
static int delta_prompt(const DeltaArgs& a, cudaStream_t st) {
    const int C = delta_channels(a), vw = a.H * a.DV;
    const bool pairs = a.D % 2 == 0 && vw % 2 == 0 && a.ldp % 2 == 0 && a.state_stride % 2 == 0 && (a.H * a.D * a.DV) % 2 == 0 &&
                       (((uintptr_t)a.proj | (uintptr_t)a.v) & (2 * sizeof(T) - 1)) == 0 &&
                       (((uintptr_t)a.qk | (uintptr_t)a.state) & 7) == 0;
#define DP_LAUNCH(NP) DP_LAUNCH_K(NP, 0)
#define DP_LAUNCH_K(NP, KF)                                                                                                    \
    do {                                                                                                                 \
        const int v_units = (vw + 64 * NP - 1) / (64 * NP);                                                              \
        dim3 grid((unsigned)((a.rows + DP_WARPS * DP_TOKENS - 1) / (DP_WARPS * DP_TOKENS)), 2 * a.G + v_units + 1);       \
        cm_launch(delta_prepare_kernel<T, NP, KF>, grid, 32 * DP_WARPS, 0, st, a, v_units, (int)pairs);                   \
    } while (0)
#define DP_CASES(NP)                            \
    do {                                        \
        if (a.K == 2) DP_LAUNCH_K(NP, 2);       \
        else if (a.K == 3) DP_LAUNCH_K(NP, 3);  \
        else if (a.K == 4) DP_LAUNCH_K(NP, 4);  \
        else DP_LAUNCH(NP);                     \
    } while (0)
    if (a.D <= 64) DP_CASES(1);
    else if (a.D <= 128) DP_CASES(2);
    else if (a.D <= 256) DP_LAUNCH(4);
    else DP_LAUNCH(16);
#undef DP_CASES
#undef DP_LAUNCH
#undef DP_LAUNCH_K
    CM_CHECK_LAUNCH();
    if (a.K > 1 && !a.from_zero) {
        cm_launch(delta_ring_kernel<T>, dim3((C + 127) / 128, a.B), 128, 0, st, a);
        CM_CHECK_LAUNCH();
    }
    if (a.chunks) return delta_chunked<T>(a, st);
    const int rc = launch_delta_scan<T>(a, st);
    if (rc != CM_OK) return rc;
    ScanArgs n = {};
    n.g = (const T*)a.proj + C;
    n.ldg = a.ldp;
    n.norm_w = a.norm_w;
    n.out = a.out;
    n.ldo = a.ldo;
    n.H = a.H;
    n.D = a.D;
    n.DV = a.DV;
    n.eps = a.eps;
    n.raw = a.raw;
    n.rows = a.rows;
    return cm_scan_norm_gate(sizeof(T) == 2 ? DT_BF16 : DT_F32, 0, n, st);
}

// Steps of any number of tokens per sequence.
extern "C" int cm_delta_prompt(int dt, const DeltaArgs* args, cudaStream_t st) {
    const DeltaArgs& a = *args;
    if (a.B <= 0 || a.rows <= 0) return CM_OK;
    const int rc = delta_check(a);
    if (rc != CM_OK) return rc;
    if (!a.gates || !a.qk || !a.v || !a.lb || !a.raw) CM_REFUSE("delta_prompt: a scratch buffer is missing");
    if (dt == DT_F32) return delta_prompt<float>(a, st);
    if (dt == DT_BF16) return delta_prompt<bf16>(a, st);
    return CM_ERR_DTYPE;
}

// ------------------------------------------------------------------------------ one token per sequence
// One block per head and sequence: filter, silu, unit vectors, both gates (their projections included), the state's step,
// norm and output gate.  Thread (column group cg, row set rs) holds four columns of the rows i = rs + RS x of S, requested
// at the very start so that they arrive under the arithmetic of the inputs.  With the old state, S^T k and S^T q are formed
// side by side (o = g S^T q + (q . k) u), so the block exchanges once.
template <typename T, int NR>
__global__ void __launch_bounds__(512)
delta_step_kernel(const DeltaArgs a, int RS) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[2][32];
    pdl_trigger();
    pdl_wait();
    const int hd = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, NT = blockDim.x, lane = tid & 31, warp = tid >> 5;
    const int D = a.D, DV = a.DV, H = a.H, G = a.G, K = a.K, kh = hd / (H / G), C = delta_channels(a);
    const long long t = a.seq_start[b];
    if (a.seq_start[b + 1] <= t) return;
    const int slot = a.seq_slot[b], pos = a.seq_pos0[b];
    const int groups = DV >> 2, cg = tid % groups, rs = tid / groups;
    float* qs = sm;                       // [D]
    float* ks = qs + ((D + 3) & ~3);      // [D]
    float* vs = ks + ((D + 3) & ~3);      // [DV]
    float* us = vs + DV;                  // [DV]
    float* pk = us + DV;                  // [RS][DV] shares of S^T k
    float* pq = pk + (size_t)RS * DV;     // [RS][DV] shares of S^T q
    float* st = delta_state(a, slot) + (long long)hd * D * DV;
    float4 S[NR];
    const bool mine = rs < RS;
#pragma unroll
    for (int x = 0; x < NR; ++x) {
        const int i = rs + RS * x;
        S[x] = mine && i < D ? *reinterpret_cast<const float4*>(st + (long long)i * DV + 4 * cg) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    // the filter over this head's q, k and v channels; the first head of a q/k head moves their ring on
    float* ring = K > 1 ? delta_ring(a, slot) : nullptr;
    const T* src = (const T*)a.proj + t * a.ldp;
    const bool own_qk = hd % (H / G) == 0;
    for (int e = tid; e < 2 * D + DV; e += NT) {
        const int c = e < D ? kh * D + e : (e < 2 * D ? G * D + kh * D + e - D : 2 * G * D + hd * DV + e - 2 * D);
        const float* w = a.taps + (long long)c * K;
        const float now = to_f32(src[c]);
        float y = 0.f;
        for (int j = 0; j < K - 1; ++j) {
            const int s = pos - K + 1 + j;
            y = fmaf(w[j], s >= 0 ? ring[(long long)(s % K) * C + c] : 0.f, y);
        }
        y = silu_f32(fmaf(w[K - 1], now, y));
        if (K > 1 && (own_qk || e >= 2 * D)) ring[(long long)(pos % K) * C + c] = now;
        if (e < D) qs[e] = y;
        else if (e < 2 * D) ks[e - D] = y;
        else vs[e - 2 * D] = rounded<T>(y);
    }
    float zb = 0.f, za = 0.f;                          // the gates' projections
    {
        const T* xr = (const T*)a.x + t * a.W;
        const T* wb = (const T*)a.w_gates + (long long)hd * a.W;
        const T* wa = (const T*)a.w_gates + (long long)(H + hd) * a.W;
        if (a.W % 8 == 0 && ((((uintptr_t)a.x) | ((uintptr_t)a.w_gates)) & 15) == 0) {
            for (int c = tid * 8; c < a.W; c += NT * 8) {
                float x[8], u[8], v[8];
                load8f<T>(xr + c, x);
                load8f<T>(wb + c, u);
                load8f<T>(wa + c, v);
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    zb = fmaf(u[i], x[i], zb);
                    za = fmaf(v[i], x[i], za);
                }
            }
        } else {
            for (int c = tid; c < a.W; c += NT) {
                const float x = to_f32(xr[c]);
                zb = fmaf(to_f32(wb[c]), x, zb);
                za = fmaf(to_f32(wa[c]), x, za);
            }
        }
        zb = warp_sum(zb);
        za = warp_sum(za);
        if (lane == 0) {
            red[0][warp] = zb;
            red[1][warp] = za;
        }
    }
    __syncthreads();
    const int nw = NT >> 5;
    zb = warp_sum(lane < nw ? red[0][lane] : 0.f);
    za = warp_sum(lane < nw ? red[1][lane] : 0.f);
    float sqq = 0.f, skk = 0.f, sqk = 0.f;             // every warp forms them for itself
    for (int i = lane; i < D; i += 32) {
        const float q = qs[i], k = ks[i];
        sqq = fmaf(q, q, sqq);
        skk = fmaf(k, k, skk);
        sqk = fmaf(q, k, sqk);
    }
    sqq = warp_sum(sqq);
    skk = warp_sum(skk);
    sqk = warp_sum(sqk);
    const float fq = a.q_scale / sqrtf(sqq + a.unit_eps), fk = 1.f / sqrtf(skk + a.unit_eps);
    const float g = expf(log_decay_of(a, hd, za)), beta = sigmoid_f32(zb), qk = sqk * fq * fk;
    if (mine) {
        float4 dk = make_float4(0.f, 0.f, 0.f, 0.f), dq = dk;
#pragma unroll
        for (int x = 0; x < NR; ++x) {
            const int i = rs + RS * x;
            if (i >= D) continue;
            const float k = ks[i], q = qs[i];
            dk.x = fmaf(S[x].x, k, dk.x); dk.y = fmaf(S[x].y, k, dk.y); dk.z = fmaf(S[x].z, k, dk.z); dk.w = fmaf(S[x].w, k, dk.w);
            dq.x = fmaf(S[x].x, q, dq.x); dq.y = fmaf(S[x].y, q, dq.y); dq.z = fmaf(S[x].z, q, dq.z); dq.w = fmaf(S[x].w, q, dq.w);
        }
        *reinterpret_cast<float4*>(pk + (size_t)rs * DV + 4 * cg) = dk;
        *reinterpret_cast<float4*>(pq + (size_t)rs * DV + 4 * cg) = dq;
    }
    __syncthreads();
    float oo = 0.f;
    for (int j = tid; j < DV; j += NT) {
        float dk = 0.f, dq = 0.f;
        for (int r = 0; r < RS; ++r) {
            dk += pk[(size_t)r * DV + j];
            dq += pq[(size_t)r * DV + j];
        }
        const float u = beta * (vs[j] - g * (dk * fk));
        const float o = fmaf(qk, u, g * (dq * fq));
        us[j] = u * fk;                                    // what meets the unscaled k below
        vs[j] = o;
        oo = fmaf(o, o, oo);
    }
    oo = warp_sum(oo);
    __syncthreads();                                       // red and us
    if (lane == 0) red[0][warp] = oo;
    if (mine) {
        const float4 u = *reinterpret_cast<const float4*>(us + 4 * cg);
#pragma unroll
        for (int x = 0; x < NR; ++x) {
            const int i = rs + RS * x;
            if (i >= D) continue;
            const float k = ks[i];
            *reinterpret_cast<float4*>(st + (long long)i * DV + 4 * cg) =
                make_float4(fmaf(k, u.x, g * S[x].x), fmaf(k, u.y, g * S[x].y), fmaf(k, u.z, g * S[x].z), fmaf(k, u.w, g * S[x].w));
        }
    }
    __syncthreads();
    const float inv = 1.f / sqrtf(warp_sum(lane < nw ? red[0][lane] : 0.f) / (float)DV + a.eps);
    for (int j = tid; j < DV; j += NT) {
        const float gz = to_f32(src[C + hd * DV + j]);
        ((T*)a.out)[t * a.ldo + (long long)hd * DV + j] = from_f32<T>(((vs[j] * inv) * a.norm_w[hd * DV + j]) * silu_f32(gz));
    }
}

static size_t delta_step_smem(int D, int DV, int rs) { return (size_t)(2 * ((D + 3) & ~3) + 2 * DV + 2 * rs * DV) * sizeof(float); }

// Threads, row sets and rows per thread of delta_step_kernel for heads of D x DV; false: it does not take them.
static bool delta_step_shape(int D, int DV, int* threads, int* rs, int* nr) {
    if (DV % 4 || DV > 1024 || D < 1) return false;
    const int groups = DV / 4;
    for (int nt = 128; nt <= 512; nt *= 2) {
        const int r = nt / groups;
        if (r < 1) continue;
        const int need = (D + r - 1) / r;
        if (need <= (nt == 512 ? 16 : 8)) {
            *threads = nt;
            *rs = r;
            *nr = need <= 4 ? 4 : (need <= 8 ? 8 : 16);
            return delta_step_smem(D, DV, r) <= 48 * 1024;
        }
    }
    return false;
}

extern "C" int cm_delta_step_fits(int D, int DV) {
    int nt, rs, nr;
    return delta_step_shape(D, DV, &nt, &rs, &nr) ? 1 : 0;
}

// Steps of exactly one token per sequence.
extern "C" int cm_delta_step(int dt, const DeltaArgs* args, cudaStream_t st) {
    const DeltaArgs& a = *args;
    if (a.B <= 0 || a.rows <= 0) return CM_OK;
    const int rc = delta_check(a);
    if (rc != CM_OK) return rc;
    int nt, rs, nr;
    if (!delta_step_shape(a.D, a.DV, &nt, &rs, &nr)) CM_REFUSE("delta_step: heads of %d x %d", a.D, a.DV);
    if (!a.x || !a.w_gates || a.W < 1) CM_REFUSE("delta_step: the mixer's input and its gate projections are missing");
    if ((((uintptr_t)a.state) & 15) || a.state_stride % 4) CM_REFUSE("delta_step: the state's rows must be 16-byte aligned");
    const size_t smem = delta_step_smem(a.D, a.DV, rs);
    dim3 grid(a.H, a.B);
#define DSTEP(TT)                                                                              \
    do {                                                                                       \
        if (nr == 4) cm_launch(delta_step_kernel<TT, 4>, grid, nt, smem, st, a, rs);           \
        else if (nr == 8) cm_launch(delta_step_kernel<TT, 8>, grid, nt, smem, st, a, rs);      \
        else cm_launch(delta_step_kernel<TT, 16>, grid, nt, smem, st, a, rs);                  \
    } while (0)
    if (dt == DT_F32) DSTEP(float);
    else if (dt == DT_BF16) DSTEP(bf16);
    else return CM_ERR_DTYPE;
#undef DSTEP
    CM_CHECK_LAUNCH();
    return CM_OK;
}
