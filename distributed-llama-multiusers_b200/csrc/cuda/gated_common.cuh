// Pieces shared by the recurrences with data-dependent gates (gated_scan.cu, delta_scan.cu): how a row's query, key and decay are
// formed, how a sequence is cut into chunks, and the scores inside a chunk under decays per channel.
#pragma once
#include "layer_common.cuh"
#include "../../../include/dllama_b200.h"

#define GC DL_GATED_CHUNK
#define GC_THREADS 256
#define GC_AS 68                  // row stride of the score matrix

enum { GATED_HEAD = 0, GATED_CHANNEL = 1, GATED_AHEAD = 2, GATED_DELTA = 3 };

__device__ __forceinline__ int gated_k_head(const DlGatedArgs& a, int h) { return a.k_heads > 0 ? h / (a.n_heads / a.k_heads) : h; }

__device__ __forceinline__ float gated_q(const DlGatedArgs& a, size_t row, int i) {
    const float v = a.q[row * a.ldq + i];
    if (!a.q_silu) return v * a.q_scale;
    float s, c;
    sigmoid_pair_f(v, s, c);
    return v * s;
}
// what a channel's gate reads besides the row: bias, lower bound, the head's rate
struct GatedChannel { float bias, lower, rate; };
__device__ __forceinline__ GatedChannel gated_channel(const DlGatedArgs& a, int h, int d) {
    GatedChannel c;
    c.bias = a.f_bias ? a.f_bias[h * a.dim + d] : 0.f;
    c.lower = a.gate == DL_GATE_LOWER ? a.lower[h * a.dim + d] : 0.f;
    c.rate = a.gate == DL_GATE_SOFTPLUS ? a.rate[h] : 0.f;
    return c;
}
// decay f from the raw gate z; with DL_GATE_LOWER also the key k
__device__ __forceinline__ void gated_form(const DlGatedArgs& a, const GatedChannel& c, float z, float& f, float& k) {
    z += c.bias;
    if (a.gate == DL_GATE_LOWER) {
        float s, t;
        sigmoid_pair_f(z, s, t);
        f = fmaf(1.f - c.lower, s, c.lower);
        k = (1.f - c.lower) * t;
    } else {
        f = a.gate == DL_GATE_ROOT_SIGMOID ? expf(-softplus_f(-z) * a.inv_tau) : a.gate == DL_GATE_EXP_EXP ? expf(-expf(z)) : expf(-c.rate * softplus_f(z));
    }
}
// decay and key of channel d of head h (its keys are those of head hk)
__device__ __forceinline__ void gated_fk(const DlGatedArgs& a, size_t row, int h, int hk, int d, float& f, float& k) {
    k = a.gate == DL_GATE_LOWER ? 0.f : a.k[row * a.ldk + hk * a.dim + d];
    gated_form(a, gated_channel(a, h, d), a.f[row * a.ldf + h * a.dim + d], f, k);
}

static inline int gated_args_ok(const DlGatedArgs& a, const char* who) {
    const bool ch = a.f != nullptr;
    if (a.n_heads < 1 || a.dim < 1 || a.vdim < 1 || a.dim > 512) { dl_set_error("%s: bad shape (heads %d, dim %d, vdim %d)", who, a.n_heads, a.dim, a.vdim); return -1; }
    if (ch && a.gate == DL_GATE_LOWER ? (!a.f_bias || !a.lower) : !a.k) { dl_set_error("%s: the gates are incomplete", who); return -1; }
    if (!ch && (!a.log_keep || !a.put || !a.den || !a.n_state)) { dl_set_error("%s: the gates are incomplete", who); return -1; }
    if (ch && ((a.gate == DL_GATE_ROOT_SIGMOID && !(a.inv_tau > 0.f)) || (a.gate == DL_GATE_SOFTPLUS && !a.rate))) { dl_set_error("%s: the gates are incomplete", who); return -1; }
    if ((a.bonus && a.beta) || (!ch && (a.bonus || a.beta || a.k_heads))) { dl_set_error("%s: these forms do not go together", who); return -1; }
    if (a.k_heads < 0 || (a.k_heads > 0 && a.n_heads % a.k_heads)) { dl_set_error("%s: %d heads on %d key heads", who, a.n_heads, a.k_heads); return -1; }
    return 0;
}

struct GatedScratch { float* S; float* dec; float* ns; };

__device__ __forceinline__ bool gated_chunk_of(const DlMambaBatch& b, int n, int c, int& row0, int& len, int& ci) {
    const int s0 = b.seq_start[n], total = b.seq_start[n + 1] - s0;
    if (c * GC >= total) return false;
    row0 = s0 + c * GC;
    len = min(GC, total - c * GC);
    ci = s0 / GC + n + c;
    return true;
}

// V columns c0 .. c0 + VW - 1 (VW: 64 or 128) of the chunk's values into [GC][VW] (zeros beyond the chunk or the head's width); a warp's
// eight rows are in flight together
template <int VW>
__device__ __forceinline__ void gated_stage_v(const DlGatedArgs& a, const int* rows, int len, int h, int c0, float* vt) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    constexpr int NRW = GC * 32 / GC_THREADS;
#pragma unroll
    for (int u = 0; u < VW / 32; ++u) {
        const int cc = lane + 32 * u;
        float v[NRW];
#pragma unroll
        for (int r = 0; r < NRW; ++r) {
            const int j = warp + r * (GC_THREADS / 32);
            v[r] = (j < len && c0 + cc < a.vdim) ? a.v[(size_t)rows[j] * a.ldv + (size_t)h * a.vdim + c0 + cc] : 0.f;
        }
#pragma unroll
        for (int r = 0; r < NRW; ++r) vt[(warp + r * (GC_THREADS / 32)) * VW + cc] = v[r];
    }
}

// keys, decays and (Q) queries of a chunk's rows into [GC][ld] each, columns [0, DP4); rows and columns that are not there: k = q = 0,
// f = 1.  COPY: the keys also into Q.  A warp's eight rows are in flight together.
template <bool WITH_Q, bool COPY>
__device__ __forceinline__ void gated_stage_rows(const DlGatedArgs& a, const int* rows, int len, int h, int hk, int DP4, int ld, float* Q, float* K, float* F) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, D = a.dim;
    constexpr int NRW = GC * 32 / GC_THREADS;
    for (int d = lane; d < DP4; d += 32) {
        float q[NRW], k[NRW], z[NRW];
        GatedChannel c = {0.f, 0.f, 0.f};
        if (d < D) c = gated_channel(a, h, d);
#pragma unroll
        for (int r = 0; r < NRW; ++r) {
            const int j = warp + r * (GC_THREADS / 32);
            const bool ok = j < len && d < D;
            const size_t row = rows[j];
            z[r] = ok ? a.f[row * a.ldf + h * D + d] : 0.f;
            k[r] = ok && a.gate != DL_GATE_LOWER ? a.k[row * a.ldk + hk * D + d] : 0.f;
            if (WITH_Q) q[r] = ok ? a.q[row * a.ldq + hk * D + d] : 0.f;
        }
#pragma unroll
        for (int r = 0; r < NRW; ++r) {
            const int j = warp + r * (GC_THREADS / 32);
            float f = 1.f;
            if (j < len && d < D) gated_form(a, c, z[r], f, k[r]);
            K[j * ld + d] = k[r];
            F[j * ld + d] = f;
            if (COPY) Q[j * ld + d] = k[r];
            if (WITH_Q) {
                float v = q[r] * a.q_scale;
                if (a.q_silu) {
                    float s, t;
                    sigmoid_pair_f(q[r], s, t);
                    v = q[r] * s;
                }
                Q[j * ld + d] = v;
            }
        }
    }
}

__device__ __forceinline__ float dot4(float4 x, float4 y, float acc) { return fmaf(x.x, y.x, fmaf(x.y, y.y, fmaf(x.z, y.z, fmaf(x.w, y.w, acc)))); }
__device__ __forceinline__ float4 mul4(float4 x, float4 y) { return make_float4(x.x * y.x, x.y * y.y, x.z * y.z, x.w * y.w); }

// Scores of a chunk's rows against its own rows, put(i, j, sum_d Q_i[d] D_ij[d] K_j[d]) for every i >= j (some i < j inside a
// sub-block are put too), D_ij[d] = product of F_t[d] over j < t <= i (AHEAD: j < t < i, and bonus[d] for i = j).  Q, K, F: [GC][DP] in
// shared memory, complete; put may write over F (every F is read before the first put).  Leaves Q_i scaled by the decay from the
// chunk's start (AHEAD: to the row before i), K_j by the decay to the end of its sub-block of 16 rows, T [4][DP] the sub-blocks'
// whole decays.  No barrier after the last writes.
template <bool AHEAD, typename Put>
__device__ __forceinline__ void decayed_scores(float* Q, float* K, const float* F, float* T, int D, int D4, int DP, const float* bonus, Put put) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tb = threadIdx.x >> 4, cb = threadIdx.x & 15;
    // inside a sub-block: for column j the running product k_j f_(j+1) .. f_i, lanes along d.  Two warps per sub-block
    // take its columns in turn; a lane's shares for all rows i are reduced together (16 values over 32 lanes).
    const int blk = warp >> 1;
    const float* Qb = Q + (size_t)blk * 16 * DP;
    const float* Kb = K + (size_t)blk * 16 * DP;
    const float* Fb = F + (size_t)blk * 16 * DP;
    float diag[8];
#pragma unroll 1
    for (int jj = 0; jj < 8; ++jj) {
        const int j = jj * 2 + (warp & 1);
        float acc[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) acc[i] = 0.f;
        for (int d = lane; d < D4; d += 32) {
            float p = Kb[j * DP + d];
#pragma unroll
            for (int i = 0; i < 16; ++i)
                if (i >= j) {
                    if (!AHEAD && i > j) p *= Fb[i * DP + d];
                    acc[i] = fmaf(Qb[i * DP + d], AHEAD && i == j ? (d < D ? bonus[d] * p : 0.f) : p, acc[i]);
                    if (AHEAD && i > j) p *= Fb[i * DP + d];
                }
        }
#pragma unroll
        for (int o = 16, m = 8; o >= 2; o >>= 1, m >>= 1) {
            const bool hi = lane & o;
#pragma unroll
            for (int t = 0; t < m; ++t) {
                const float keep = hi ? acc[t + m] : acc[t], send = hi ? acc[t] : acc[t + m];
                acc[t] = keep + __shfl_xor_sync(0xffffffffu, send, o);
            }
        }
        acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], 1);
        // this lane now holds row i = lane / 2 of column j
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (u == jj) diag[u] = acc[0];
    }
    __syncthreads();
    // rows scaled by the decay from their block's start (Q) / to their block's end (K); T: a block's whole decay
    for (int t = threadIdx.x; t < 4 * D4; t += GC_THREADS) {
        const int bk = t / D4, d = t - bk * D4;
        float p = 1.f;
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            if (AHEAD) Q[(bk * 16 + i) * DP + d] *= p;
            p *= F[(bk * 16 + i) * DP + d];
            if (!AHEAD) Q[(bk * 16 + i) * DP + d] *= p;
        }
        T[bk * DP + d] = p;
        p = 1.f;
#pragma unroll
        for (int i = 15; i >= 0; --i) {
            K[(bk * 16 + i) * DP + d] *= p;
            p *= F[(bk * 16 + i) * DP + d];
        }
    }
    __syncthreads();
    // between sub-blocks: thread (i, j) = (tb, cb) of the six block pairs
    float a10 = 0.f, a20 = 0.f, a21 = 0.f, a30 = 0.f, a31 = 0.f, a32 = 0.f;
    for (int d = 0; d < D4; d += 4) {
        const float4 q1 = *reinterpret_cast<const float4*>(Q + (16 + tb) * DP + d), q2 = *reinterpret_cast<const float4*>(Q + (32 + tb) * DP + d);
        const float4 q3 = *reinterpret_cast<const float4*>(Q + (48 + tb) * DP + d);
        const float4 k0 = *reinterpret_cast<const float4*>(K + cb * DP + d), k1 = *reinterpret_cast<const float4*>(K + (16 + cb) * DP + d);
        const float4 k2 = *reinterpret_cast<const float4*>(K + (32 + cb) * DP + d);
        const float4 t1 = *reinterpret_cast<const float4*>(T + DP + d), t2 = *reinterpret_cast<const float4*>(T + 2 * DP + d);
        const float4 k0t = mul4(k0, t1), k1t = mul4(k1, t2);
        a10 = dot4(q1, k0, a10);
        a21 = dot4(q2, k1, a21);
        a32 = dot4(q3, k2, a32);
        a20 = dot4(q2, k0t, a20);
        a31 = dot4(q3, k1t, a31);
        a30 = dot4(q3, mul4(k0t, t2), a30);
    }
    __syncthreads();                          // F is done with: the scores may take its place
    put(16 + tb, cb, a10);
    put(32 + tb, cb, a20);
    put(32 + tb, 16 + cb, a21);
    put(48 + tb, cb, a30);
    put(48 + tb, 16 + cb, a31);
    put(48 + tb, 32 + cb, a32);
#pragma unroll
    for (int jj = 0; jj < 8; ++jj) {
        const int j = jj * 2 + (warp & 1), i = lane >> 1;
        if ((lane & 1) == 0) put(blk * 16 + i, blk * 16 + j, diag[jj]);
    }
    // Q: the decay from the chunk's start
    for (int t = threadIdx.x; t < 3 * D4; t += GC_THREADS) {
        const int bk = t / D4 + 1, d = t - (bk - 1) * D4;
        float p = T[d];
        for (int u = 1; u < bk; ++u) p *= T[u * DP + d];
#pragma unroll
        for (int i = 0; i < 16; ++i) Q[(bk * 16 + i) * DP + d] *= p;
    }
}

int gated_chunk_out_channel(const DlMambaBatch& b, int n_seq, int max_chunks, const DlGatedArgs& a, const GatedScratch& sc, cudaStream_t st);
