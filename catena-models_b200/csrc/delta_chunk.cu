// Prompt form of the gated delta rule (delta.cu): the same recurrence regrouped into chunks of 64 rows, so that what runs
// one after the other is one small product per chunk instead of one step per row.
//
// Rows t, s of a chunk, L_t the sum of the log decays up to and with row t, S the state before the chunk.  Unrolled, the
// corrections u_t of the chunk satisfy a unit lower triangular system,
//
//   u_t + sum_(s<t) A_ts u_s = beta_t (v_t - e^(L_t) S^T k_t)        A_ts = beta_t e^(L_t - L_s) (k_t . k_s)
//
// so with (I + A) [W | U] = [beta e^L K | beta V] the corrections are U - W S, and everything the chunk does is linear in S:
//
//   state after the chunk    M S + N      M = e^(L_n) I - K~^T W,   N = K~^T U       (K~_s = e^(L_n - L_s) k_s)
//   outputs                  Q' S + O     Q' = diag(e^L) Q - P W,   O = P U          (P_ts = e^(L_t - L_s) (q_t . k_s), s <= t)
//
// Pass 1 forms M, N, Q' and O of every chunk (all side by side; the system is solved by substitution, a thread per
// column); pass 2 walks S <- M S + N and leaves the state before every chunk; pass 3 adds Q' S to O, and applies the unit
// norm, the channel weights and the output gate.  All of it is float on the CUDA cores: products of 4 x 4 register tiles
// out of shared memory.  Exponents are of sums of log decays over later rows, so none is positive.
#include "common.cuh"
#include "delta.h"
#include <math.h>

#define DC 64                    // rows of a chunk
#define DC_THREADS 256
#define DC_LD 68                 // pitch of the 64-column operands: float4 rows, neighbouring rows four banks apart
#define DC_COLS 8                // columns of the state that a block of pass 2 owns

struct DeltaChunkGeom {
    int D4, DV4;                 // D and DV rounded up to multiples of 4
    int chunks;                  // chunks per sequence that the launch provides for
    int NCp;                     // pitch of [W | U]
    int stages;                  // chunks whose M^T and N pass 2 holds at a time
    long long stride;            // floats of one chunk of one head in the scratch: M^T [D4][D4], N [D4][DV4], Q'^T [D4][DC]
};

static __host__ __device__ __forceinline__ constexpr int dc_stages(int D4) { return D4 <= 64 ? 4 : (D4 <= 96 ? 3 : 2); }
static __host__ __device__ __forceinline__ DeltaChunkGeom delta_chunk_geom(int D, int DV, int max_len) {
    DeltaChunkGeom g;
    g.D4 = (D + 3) & ~3;
    g.DV4 = (DV + 3) & ~3;
    g.chunks = (max_len + DC - 1) / DC;
    g.NCp = g.D4 + g.DV4 + 4;
    g.stages = dc_stages(g.D4);
    g.stride = (long long)g.D4 * (g.D4 + g.DV4 + DC);
    return g;
}
static size_t delta_chunk_smem(const DeltaChunkGeom& g) {
    const size_t first = 2 * (size_t)g.D4 * DC_LD, x = (size_t)DC * g.NCp;
    return ((first > x ? first : x) + (size_t)DC * (g.D4 + 4) + 2 * DC * DC_LD + 4 * DC) * sizeof(float);
}
static size_t delta_walk_smem(const DeltaChunkGeom& g) {
    return ((size_t)g.stages * g.D4 * (g.D4 + 4 + DC_COLS) + 2 * (size_t)g.D4 * DC_COLS) * sizeof(float);
}
static size_t delta_read_smem(const DeltaChunkGeom& g) { return ((size_t)g.D4 * DC_LD + (size_t)g.D4 * DC_LD) * sizeof(float); }

__device__ __forceinline__ float* delta_chunk_at(const DeltaArgs& a, const DeltaChunkGeom& g, int b, int hd, int c) {
    return a.chunks + (((long long)b * a.H + hd) * g.chunks + c) * g.stride;
}

// acc[i][j] += sum over k in [k0, k1) of A[k][i] B[k][j], four rows and four columns from float4 rows
__device__ __forceinline__ void tile_mac(float (&acc)[4][4], const float* A, int lda, const float* B, int ldb, int k0, int k1) {
#pragma unroll 4
    for (int k = k0; k < k1; ++k) {
        const float4 x = *reinterpret_cast<const float4*>(A + (size_t)k * lda), y = *reinterpret_cast<const float4*>(B + (size_t)k * ldb);
        const float xs[4] = {x.x, x.y, x.z, x.w}, ys[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xs[i], ys[j], acc[i][j]);
    }
}
// two sums at once: u += a w, v += b w (one instruction on register pairs)
__device__ __forceinline__ void fma_two(float& u, float& v, float a, float b, float w) {
    asm("{\n\t.reg .b64 p, q, r;\n\tmov.b64 p, {%0, %1};\n\tmov.b64 q, {%2, %3};\n\tmov.b64 r, {%4, %4};\n\t"
        "fma.rn.f32x2 p, q, r, p;\n\tmov.b64 {%0, %1}, p;\n\t}"
        : "+f"(u), "+f"(v) : "f"(a), "f"(b), "f"(w));
}
__device__ __forceinline__ void tile_zero(float (&acc)[4][4]) {
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
}

// ------------------------------------------------------------------------------ pass 1
// DK, DVK: the heads' sizes where they are known to the compiler (multiples of 4), or 0.
template <typename T, int DK, int DVK>
__global__ void __launch_bounds__(DC_THREADS, 2)
delta_chunk_kernel(const DeltaArgs a, const DeltaChunkGeom g) {
    extern __shared__ __align__(16) float sm[];
    pdl_wait();
    const int c = blockIdx.x, hd = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
    const int s0 = a.seq_start[b], s1 = a.seq_start[b + 1];
    const long long r0 = (long long)s0 + (long long)c * DC;
    const int n = (int)min((long long)DC, s1 - r0);
    if (n <= 0) return;
    const int D = DK ? DK : a.D, DV = DVK ? DVK : a.DV, D4 = DK ? DK : g.D4, DV4 = DVK ? DVK : g.DV4;
    const int H = a.H, G = a.G, kh = hd / (H / G), NC = D4 + DV4, NCp = NC + 4, ldk = D4 + 4;
    const size_t first = 2 * (size_t)D4 * DC_LD, xsz = (size_t)DC * NCp;
    float* kT = sm;                                     // [D4][DC_LD]: k_t,i at [i][t]
    float* qT = kT + (size_t)D4 * DC_LD;                // the same of q
    float* X = sm;                                      // [DC][NCp]: [W | U], over kT and qT once they are done with
    float* kr = sm + (first > xsz ? first : xsz);       // [DC][ldk]: k_t,i at [t][i]
    float* AT = kr + (size_t)DC * ldk;                  // [DC][DC_LD]: A_ts at [s][t]
    float* PT = AT + DC * DC_LD;                        // P_ts at [s][t]
    float* cl = PT + DC * DC_LD;                        // [DC]: L_t
    float* be = cl + DC;                                // beta_t
    float* ga = be + DC;                                // e^(L_t)
    float* de = ga + DC;                                // e^(L_n - L_t)
    const long long ldqk = 2LL * G * D;
    const float* Q = a.qk + r0 * ldqk + (long long)kh * D;
    const float* K = Q + (long long)G * D;
    const bool vec = D % 4 == 0 && (((uintptr_t)a.qk) & 15) == 0;
    for (int e = tid; e < DC * (D4 >> 2); e += DC_THREADS) {
        const int r = e % DC, i = (e / DC) * 4;
        float k[4] = {}, q[4] = {};
        if (r < n) {
            if (vec) {
                const float4 kk = *reinterpret_cast<const float4*>(K + r * ldqk + i), qq = *reinterpret_cast<const float4*>(Q + r * ldqk + i);
                k[0] = kk.x; k[1] = kk.y; k[2] = kk.z; k[3] = kk.w;
                q[0] = qq.x; q[1] = qq.y; q[2] = qq.z; q[3] = qq.w;
            } else {
                for (int x = 0; x < 4; ++x)
                    if (i + x < D) {
                        k[x] = K[r * ldqk + i + x];
                        q[x] = Q[r * ldqk + i + x];
                    }
            }
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            kT[(size_t)(i + x) * DC_LD + r] = k[x];
            qT[(size_t)(i + x) * DC_LD + r] = q[x];
        }
        *reinterpret_cast<float4*>(kr + (size_t)r * ldk + i) = make_float4(k[0], k[1], k[2], k[3]);
    }
    if (tid < 32) {                                     // running sums of the log decays: two rows a lane
        const int ra = 2 * tid, rb = ra + 1;
        const float la = ra < n ? a.lb[(r0 + ra) * 2 * H + hd] : 0.f, lb = rb < n ? a.lb[(r0 + rb) * 2 * H + hd] : 0.f;
        float run = la + lb;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, run, o);
            if (tid >= o) run += up;
        }
        const float total = __shfl_sync(0xffffffffu, run, 31), before = run - (la + lb);
        const float ca = before + la, cb = ca + lb;
        cl[ra] = ca;
        cl[rb] = cb;
        ga[ra] = expf(ca);
        ga[rb] = expf(cb);
        de[ra] = expf(fminf(total - ca, 0.f));
        de[rb] = expf(fminf(total - cb, 0.f));
        be[ra] = ra < n ? a.lb[(r0 + ra) * 2 * H + H + hd] : 0.f;
        be[rb] = rb < n ? a.lb[(r0 + rb) * 2 * H + H + hd] : 0.f;
    }
    __syncthreads();
    const int ty = tid >> 4, tx = tid & 15;             // a thread's tile: rows 4 ty .., columns 4 tx .. of a 64 x 64 piece
    {
        float kk[4][4], qk[4][4];
        tile_zero(kk);
        tile_zero(qk);
        const int t = 4 * ty, s = 4 * tx;
        if (s <= t + 3)
#pragma unroll 2
            for (int i = 0; i < D4; ++i) {
                const float4 kt = *reinterpret_cast<const float4*>(kT + (size_t)i * DC_LD + t);
                const float4 qt = *reinterpret_cast<const float4*>(qT + (size_t)i * DC_LD + t);
                const float4 ks = *reinterpret_cast<const float4*>(kT + (size_t)i * DC_LD + s);
                const float x[4] = {kt.x, kt.y, kt.z, kt.w}, y[4] = {qt.x, qt.y, qt.z, qt.w}, z[4] = {ks.x, ks.y, ks.z, ks.w};
#pragma unroll
                for (int u = 0; u < 4; ++u)
#pragma unroll
                    for (int v = 0; v < 4; ++v) {
                        kk[u][v] = fmaf(x[u], z[v], kk[u][v]);
                        qk[u][v] = fmaf(y[u], z[v], qk[u][v]);
                    }
            }
#pragma unroll
        for (int v = 0; v < 4; ++v) {
            float A[4], P[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const float f = s + v <= t + u ? expf(fminf(cl[t + u] - cl[s + v], 0.f)) : 0.f;
                A[u] = s + v < t + u ? be[t + u] * f * kk[u][v] : 0.f;
                P[u] = f * qk[u][v];
            }
            *reinterpret_cast<float4*>(AT + (size_t)(s + v) * DC_LD + t) = make_float4(A[0], A[1], A[2], A[3]);
            *reinterpret_cast<float4*>(PT + (size_t)(s + v) * DC_LD + t) = make_float4(P[0], P[1], P[2], P[3]);
        }
    }
    __syncthreads();                                    // A and P are complete; kT and qT are done with
    // (I + A) x = column of [beta e^L K | beta V]: once x_s is final it leaves the rows below
    for (int col = tid; col < NC; col += DC_THREADS) {
        float x[DC];
        if (col < D4) {
#pragma unroll
            for (int r = 0; r < DC; ++r) x[r] = be[r] * ga[r] * kr[(size_t)r * ldk + col];
        } else {
            const int j = col - D4;
            const T* V = (const T*)a.v + r0 * ((long long)H * DV) + (long long)hd * DV + j;
#pragma unroll
            for (int r = 0; r < DC; ++r) x[r] = r < n && j < DV ? be[r] * to_f32(V[(long long)r * H * DV]) : 0.f;
        }
#pragma unroll
        for (int s = 0; s < DC - 1; ++s) {
            const float xs = -x[s];
#pragma unroll
            for (int t = (s + 1) & ~3; t < DC; t += 4) {                // A_ts is zero for t <= s
                const float4 A = *reinterpret_cast<const float4*>(AT + s * DC_LD + t);
                fma_two(x[t], x[t + 1], A.x, A.y, xs);
                fma_two(x[t + 2], x[t + 3], A.z, A.w, xs);
            }
        }
#pragma unroll
        for (int r = 0; r < DC; ++r) X[(size_t)r * NCp + col] = x[r];
    }
    __syncthreads();
    for (int e = tid; e < DC * D4; e += DC_THREADS) {   // K~
        const int r = e / D4, i = e - r * D4;
        kr[(size_t)r * ldk + i] *= de[r];
    }
    __syncthreads();
    pdl_trigger();                                      // not before: waiting blocks of the next pass would take this one's room
    float* MT = delta_chunk_at(a, g, b, hd, c);
    float* N = MT + (size_t)D4 * D4;
    float* QT = N + (size_t)D4 * DV4;
    const float total = ga[DC - 1];                     // rows past n add no decay
    float acc[4][4];
    for (int i0 = 4 * ty; i0 < D4; i0 += 64) {
        for (int j0 = 4 * tx; j0 < D4; j0 += 64) {      // M^T: rows are the columns of W
            tile_zero(acc);
            tile_mac(acc, X + i0, NCp, kr + j0, ldk, 0, n);
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                float o[4];
#pragma unroll
                for (int v = 0; v < 4; ++v) o[v] = (i0 + u == j0 + v ? total : 0.f) - acc[u][v];
                *reinterpret_cast<float4*>(MT + (size_t)(i0 + u) * D4 + j0) = make_float4(o[0], o[1], o[2], o[3]);
            }
        }
        for (int j0 = 4 * tx; j0 < DV4; j0 += 64) {     // N
            tile_zero(acc);
            tile_mac(acc, kr + i0, ldk, X + D4 + j0, NCp, 0, n);
#pragma unroll
            for (int u = 0; u < 4; ++u)
                *reinterpret_cast<float4*>(N + (size_t)(i0 + u) * DV4 + j0) = make_float4(acc[u][0], acc[u][1], acc[u][2], acc[u][3]);
        }
        {                                               // Q'^T: rows are the columns of W, columns the rows of the chunk
            const int t = 4 * tx;
            tile_zero(acc);
            tile_mac(acc, X + i0, NCp, PT + t, DC_LD, 0, min(n, t + 4));
            float q[4][4];
#pragma unroll
            for (int v = 0; v < 4; ++v)
#pragma unroll
                for (int u = 0; u < 4; ++u) q[u][v] = t + v < n && i0 + u < D ? Q[(t + v) * ldqk + i0 + u] * ga[t + v] : 0.f;
#pragma unroll
            for (int u = 0; u < 4; ++u)
                *reinterpret_cast<float4*>(QT + (size_t)(i0 + u) * DC + t) =
                    make_float4(q[u][0] - acc[u][0], q[u][1] - acc[u][1], q[u][2] - acc[u][2], q[u][3] - acc[u][3]);
        }
    }
    for (int j0 = 4 * tx; j0 < DV4; j0 += 64) {         // O
        const int t = 4 * ty;
        tile_zero(acc);
        tile_mac(acc, PT + t, DC_LD, X + D4 + j0, NCp, 0, min(n, t + 4));
#pragma unroll
        for (int u = 0; u < 4; ++u)
            if (t + u < n) {
                float* o = a.raw + (r0 + t + u) * ((long long)H * DV) + (long long)hd * DV + j0;
#pragma unroll
                for (int v = 0; v < 4; ++v)
                    if (j0 + v < DV) o[v] = acc[u][v];
            }
    }
}

// ------------------------------------------------------------------------------ pass 2
__device__ __forceinline__ void dc_copy16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// A block owns DC_COLS columns of one head's S for one sequence.  S lies in shared memory, twice (the state before and
// behind the present chunk); M^T and N of the next chunks are on their way while the present one is multiplied (several
// chunks ahead where shared memory allows).  A tile of 4 x 4 outputs belongs to PARTS neighbouring lanes, of which lane
// `part` takes the inner channels part, part + PARTS, ...; their shares are exchanged by shuffles in halves (every lane ends
// with 16 / PARTS of the outputs), so a chunk takes one barrier.  N's place receives the state before the chunk.
template <int PARTS, int DK>
__global__ void __launch_bounds__(DC_THREADS)
delta_walk_kernel(const DeltaArgs a, const DeltaChunkGeom g) {
    extern __shared__ __align__(16) float sm[];
    pdl_wait();
    const int hd = blockIdx.x, b = blockIdx.z, tid = threadIdx.x, j0 = blockIdx.y * DC_COLS;
    const int s0 = a.seq_start[b], rows = a.seq_start[b + 1] - s0;
    if (rows <= 0) return;
    const int D = DK ? DK : a.D, DV = a.DV, D4 = DK ? DK : g.D4, DV4 = g.DV4, ldm = D4 + 4, chunks = (rows + DC - 1) / DC;
    const int stages = DK ? dc_stages(DK) : g.stages;
    const int m_floats = D4 * ldm, n_floats = D4 * DC_COLS;
    float* Ms = sm;                                     // [stages][D4][ldm]
    float* Ns = Ms + stages * (size_t)m_floats;         // [stages][D4][DC_COLS]
    float* S = Ns + stages * (size_t)n_floats;          // [2][D4][DC_COLS]
    float* st = a.state + (long long)a.seq_slot[b] * a.state_stride + (long long)hd * D * DV;
    float* chunk = delta_chunk_at(a, g, b, hd, 0);
    const int quads = D4 / 4;
    auto fetch = [&](int c, int slot) {                 // one group of copies per call, empty past the last chunk
        if (c < chunks) {
            const float* M = chunk + c * g.stride;
            const float* N = M + (size_t)D4 * D4;
            float* md = Ms + (size_t)slot * m_floats;
            float* nd = Ns + (size_t)slot * n_floats;
            for (int k = tid >> 4; k < D4; k += DC_THREADS / 16)
                for (int x = tid & 15; x < quads; x += 16) dc_copy16(md + k * ldm + 4 * x, M + k * D4 + 4 * x);
            for (int e = tid; e < D4 * (DC_COLS / 4); e += DC_THREADS) {
                const int i = e / (DC_COLS / 4), j = 4 * (e % (DC_COLS / 4));
                if (j0 + j < DV4) dc_copy16(nd + i * DC_COLS + j, N + (size_t)i * DV4 + j0 + j);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (int c = 0; c + 1 < stages; ++c) fetch(c, c);
    for (int e = tid; e < n_floats; e += DC_THREADS) {
        const int i = e / DC_COLS, j = j0 + e % DC_COLS;
        S[e] = i < D && j < DV ? st[(long long)i * DV + j] : 0.f;
    }
    for (int e = tid; e < stages * n_floats; e += DC_THREADS)            // columns past DV4 are never fetched
        if (j0 + e % DC_COLS >= DV4) Ns[e] = 0.f;
    constexpr int CT = DC_COLS / 4;                     // column tiles
    constexpr int OWN = PARTS >= 16 ? 1 : 16 / PARTS;   // outputs of the tile that a lane ends with
    const int part = tid % PARTS, tile = tid / PARTS, i0 = 4 * (tile / CT), jt = 4 * (tile % CT);
    const bool mine = tile < quads * CT;
    const unsigned everyone = 0xffffffffu;
    // which outputs (4 x row + column within the tile) the halving leaves with this lane: the first exchange decides the
    // highest bit
    int own = 0;
#pragma unroll
    for (int o = PARTS / 2, half = 8; o > 0 && half > 0; o >>= 1, half >>= 1) own += (part & o) ? half : 0;
    const bool writer = mine && (PARTS < 32 || !(part & 1));
    int slot = 0;
    for (int c = 0; c < chunks; ++c) {
        if (stages == 4) asm volatile("cp.async.wait_group 2;" ::: "memory");
        else if (stages == 3) asm volatile("cp.async.wait_group 1;" ::: "memory");
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                // chunk c is here, S is complete, the slot of the chunk before is free
        fetch(c + stages - 1, slot == 0 ? stages - 1 : slot - 1);
        const float* M = Ms + (size_t)slot * m_floats;
        const float* N = Ns + (size_t)slot * n_floats;
        const float* Sb = S + (c & 1) * n_floats;
        float* Sa = S + ((c + 1) & 1) * n_floats;
        float v[16];
        {
            float acc[4][4];
            tile_zero(acc);
            if (mine) {
#pragma unroll 4
                for (int k = part; k < D4; k += PARTS) {
                    const float4 x = *reinterpret_cast<const float4*>(M + k * ldm + i0), y = *reinterpret_cast<const float4*>(Sb + k * DC_COLS + jt);
                    const float xs[4] = {x.x, x.y, x.z, x.w}, ys[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i)
#pragma unroll
                        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xs[i], ys[j], acc[i][j]);
                }
            }
#pragma unroll
            for (int e = 0; e < 16; ++e) v[e] = acc[e >> 2][e & 3];
        }
#pragma unroll
        for (int o = PARTS / 2, half = 8; o > 0; o >>= 1, half >>= 1) {
            const bool up = part & o;
            if (half > 0) {
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    if (e >= half) break;
                    const float give = up ? v[e] : v[e + half], keep = up ? v[e + half] : v[e];
                    v[e] = keep + __shfl_xor_sync(everyone, give, o);
                }
            } else {
                v[0] += __shfl_xor_sync(everyone, v[0], o);
            }
        }
        if (writer) {
            float* before = chunk + c * g.stride + (size_t)D4 * D4;
#pragma unroll
            for (int e = 0; e < OWN; ++e) {
                const int out = own + e, i = i0 + (out >> 2), j = jt + (out & 3), at = i * DC_COLS + j;
                if (j0 + j < DV4) before[(size_t)i * DV4 + j0 + j] = Sb[at];
                Sa[at] = v[e] + N[at];
            }
        }
        slot = slot + 1 == stages ? 0 : slot + 1;
    }
    pdl_trigger();
    __syncthreads();
    const float* Se = S + (chunks & 1) * n_floats;
    for (int e = tid; e < n_floats; e += DC_THREADS) {
        const int i = e / DC_COLS, j = j0 + e % DC_COLS;
        if (i < D && j < DV) st[(long long)i * DV + j] = Se[e];
    }
}

// ------------------------------------------------------------------------------ pass 3
// four elements from p on as floats, of which `left` exist (zeros behind them); `vec`: one access
__device__ __forceinline__ void load_four(float* out, const float* p, int left, bool vec) {
    if (vec && left > 0) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        out[0] = t.x; out[1] = t.y; out[2] = t.z; out[3] = t.w;
    } else {
#pragma unroll
        for (int v = 0; v < 4; ++v) out[v] = v < left ? p[v] : 0.f;
    }
}
__device__ __forceinline__ void load_four(float* out, const bf16* p, int left, bool vec) {
    if (vec && left > 0) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
        const float2 x = __bfloat1622float2(h[0]), y = __bfloat1622float2(h[1]);
        out[0] = x.x; out[1] = x.y; out[2] = y.x; out[3] = y.y;
    } else {
#pragma unroll
        for (int v = 0; v < 4; ++v) out[v] = v < left ? __bfloat162float(p[v]) : 0.f;
    }
}

// A block takes the 64 rows of a chunk of one head: o = O + Q' S, then the unit norm over the head's channels, the channel
// weights and the gate's silu.  NT pieces of 64 columns; the sixteen threads of a row's columns are half a warp.
template <typename T, int NT, int DK>
__global__ void __launch_bounds__(DC_THREADS)
delta_read_kernel(const DeltaArgs a, const DeltaChunkGeom g) {
    extern __shared__ __align__(16) float sm[];
    pdl_wait();
    const int c = blockIdx.x, hd = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
    const long long r0 = (long long)a.seq_start[b] + (long long)c * DC;
    const int n = (int)min((long long)DC, a.seq_start[b + 1] - r0);
    if (n <= 0) return;
    const int DV = a.DV, D4 = DK ? DK : g.D4, DV4 = g.DV4, H = a.H, ty = tid >> 4, tx = tid & 15, t = 4 * ty;
    float* Qs = sm;                                     // [D4][DC_LD]: Q'^T
    float* Ss = Qs + (size_t)D4 * DC_LD;                // [D4][DC_LD]: 64 columns of the state before the chunk
    const float* S = delta_chunk_at(a, g, b, hd, c) + (size_t)D4 * D4;
    const float* QT = S + (size_t)D4 * DV4;
    for (int e = tid; e < D4 * (DC / 4); e += DC_THREADS) {
        const int i = e / (DC / 4), x = 4 * (e - i * (DC / 4));
        *reinterpret_cast<float4*>(Qs + (size_t)i * DC_LD + x) = *reinterpret_cast<const float4*>(QT + (size_t)i * DC + x);
    }
    // four neighbouring channels as one access: every head, pitch and base a multiple of four elements
    const bool vec = DV % 4 == 0 && a.ldp % 4 == 0 && a.ldo % 4 == 0 && (2 * a.G * a.D) % 4 == 0 &&
                     (((uintptr_t)a.proj | (uintptr_t)a.out) & (4 * sizeof(T) - 1)) == 0 && (((uintptr_t)a.raw | (uintptr_t)a.norm_w) & 15) == 0;
    float o[NT][4][4];
    float ss[4] = {0.f, 0.f, 0.f, 0.f};
    const long long ldr = (long long)H * DV;
#pragma unroll
    for (int p = 0; p < NT; ++p) {
        __syncthreads();                                // Q' is here; the piece before is no longer read
        for (int e = tid; e < D4 * 16; e += DC_THREADS) {
            const int i = e >> 4, x = 4 * (e & 15), j = 64 * p + x;
            *reinterpret_cast<float4*>(Ss + (size_t)i * DC_LD + x) =
                j < DV4 ? *reinterpret_cast<const float4*>(S + (size_t)i * DV4 + j) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        __syncthreads();
        const int j0 = 64 * p + 4 * tx;
#pragma unroll
        for (int u = 0; u < 4; ++u) load_four(o[p][u], a.raw + (r0 + t + u) * ldr + (long long)hd * DV + j0, t + u < n ? DV - j0 : 0, vec);
        tile_mac(o[p], Qs + t, DC_LD, Ss + 4 * tx, DC_LD, 0, D4);
#pragma unroll
        for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int v = 0; v < 4; ++v) ss[u] = fmaf(o[p][u][v], o[p][u][v], ss[u]);
    }
    pdl_trigger();
    const int C = 2 * a.G * a.D + H * DV;
#pragma unroll
    for (int u = 0; u < 4; ++u) {
#pragma unroll
        for (int x = 8; x > 0; x >>= 1) ss[u] += __shfl_xor_sync(0xffffffffu, ss[u], x);
        if (t + u >= n) continue;
        const float inv = 1.f / sqrtf(ss[u] / (float)DV + a.eps);
        const T* G = (const T*)a.proj + (r0 + t + u) * a.ldp + C + (long long)hd * DV;
        T* O = (T*)a.out + (r0 + t + u) * a.ldo + (long long)hd * DV;
#pragma unroll
        for (int p = 0; p < NT; ++p) {
            const int j0 = 64 * p + 4 * tx;
            float gz[4], w[4], y[4];
            load_four(gz, G + j0, DV - j0, vec);
            load_four(w, a.norm_w + hd * DV + j0, DV - j0, vec);
#pragma unroll
            for (int v = 0; v < 4; ++v) y[v] = ((o[p][u][v] * inv) * w[v]) * (gz[v] * sigmoid_f32(gz[v]));
            if (vec && j0 < DV) {
                if constexpr (sizeof(T) == 2) {
                    uint2 raw;
                    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
                    h[0] = __floats2bfloat162_rn(y[0], y[1]);
                    h[1] = __floats2bfloat162_rn(y[2], y[3]);
                    *reinterpret_cast<uint2*>(O + j0) = raw;
                } else {
                    *reinterpret_cast<float4*>(O + j0) = make_float4(y[0], y[1], y[2], y[3]);
                }
            } else {
                for (int v = 0; v < 4; ++v)
                    if (j0 + v < DV) O[j0 + v] = from_f32<T>(y[v]);
            }
        }
    }
}

// Floats of scratch that the chunked form takes, or 0 if it does not take heads of D x DV.
extern "C" long long cm_delta_chunk_floats(int B, int max_len, int H, int D, int DV) {
    if (D < 1 || DV < 1 || D > 128 || DV > 256 || B < 1 || max_len < 1) return 0;
    const DeltaChunkGeom g = delta_chunk_geom(D, DV, max_len);
    if (delta_chunk_smem(g) > 220 * 1024 || delta_walk_smem(g) > 220 * 1024) return 0;
    return (long long)B * H * g.chunks * g.stride;
}

template <typename T>
int delta_chunked(const DeltaArgs& a, cudaStream_t st) {
    const DeltaChunkGeom g = delta_chunk_geom(a.D, a.DV, a.max_len);
    if (cm_delta_chunk_floats(a.B, a.max_len, a.H, a.D, a.DV) <= 0) CM_REFUSE("delta_chunked: heads of %d x %d", a.D, a.DV);
    const size_t s1 = delta_chunk_smem(g), s2 = delta_walk_smem(g), s3 = delta_read_smem(g);
    // lanes per tile of pass 2: as many as the block's threads give every tile (64 tiles at most)
    const int tiles = g.D4 / 4 * (DC_COLS / 4);
    auto walk = a.D == 64    ? delta_walk_kernel<8, 64>
                : a.D == 128 ? delta_walk_kernel<4, 128>
                : tiles <= 8 ? delta_walk_kernel<32, 0>
                : tiles <= 16 ? delta_walk_kernel<16, 0>
                : tiles <= 32 ? delta_walk_kernel<8, 0>
                              : delta_walk_kernel<4, 0>;
    auto first = delta_chunk_kernel<T, 0, 0>;
    if constexpr (sizeof(T) == 2) {
        if (a.D == 64 && a.DV == 64) first = delta_chunk_kernel<T, 64, 64>;
        else if (a.D == 64 && a.DV == 128) first = delta_chunk_kernel<T, 64, 128>;
        else if (a.D == 128 && a.DV == 128) first = delta_chunk_kernel<T, 128, 128>;
    }
    if (cudaFuncSetAttribute(first, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1) != cudaSuccess ||
        cudaFuncSetAttribute(walk, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2) != cudaSuccess) {
        cudaGetLastError();
        CM_REFUSE("delta_chunked: %zu and %zu bytes of shared memory refused", s1, s2);
    }
    cm_launch(first, dim3(g.chunks, a.H, a.B), DC_THREADS, s1, st, a, g);
    CM_CHECK_LAUNCH();
    // in plain stream order, so that its blocks spread evenly over the SMs (see launch_delta_scan)
    cm_launch_cluster(walk, dim3(a.H, (a.DV + DC_COLS - 1) / DC_COLS, a.B), DC_THREADS, s2, st, 1, false, a, g);
    CM_CHECK_LAUNCH();
#define DC_READ(NT)                          \
    do {                                     \
        if (a.D == 64) DC_READ_D(NT, 64);    \
        else if (a.D == 128) DC_READ_D(NT, 128); \
        else DC_READ_D(NT, 0);               \
    } while (0)
#define DC_READ_D(NT, DK)                                                                                                       \
    do {                                                                                                                  \
        cudaFuncSetAttribute(delta_read_kernel<T, NT, DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s3);             \
        cm_launch(delta_read_kernel<T, NT, DK>, dim3(g.chunks, a.H, a.B), DC_THREADS, s3, st, a, g);                          \
    } while (0)
    if (a.DV <= 64) DC_READ(1);
    else if (a.DV <= 128) DC_READ(2);
    else if (a.DV <= 192) DC_READ(3);
    else DC_READ(4);
#undef DC_READ
#undef DC_READ_D
    CM_CHECK_LAUNCH();
    return CM_OK;
}
template int delta_chunked<float>(const DeltaArgs&, cudaStream_t);
template int delta_chunked<bf16>(const DeltaArgs&, cudaStream_t);
