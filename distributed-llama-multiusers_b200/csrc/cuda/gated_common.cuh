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
// decay and key of channel d of head h (its keys are those of head hk)
__device__ __forceinline__ void gated_fk(const DlGatedArgs& a, size_t row, int h, int hk, int d, float& f, float& k) {
    const int i = h * a.dim + d;
    float z = a.f[row * a.ldf + i];
    if (a.f_bias) z += a.f_bias[i];
    if (a.gate == DL_GATE_LOWER) {
        float s, c;
        sigmoid_pair_f(z, s, c);
        const float l = a.lower[i];
        f = fmaf(1.f - l, s, l);
        k = (1.f - l) * c;
        return;
    }
    k = a.k[row * a.ldk + hk * a.dim + d];
    f = a.gate == DL_GATE_ROOT_SIGMOID ? expf(-softplus_f(-z) * a.inv_tau) : a.gate == DL_GATE_EXP_EXP ? expf(-expf(z)) : expf(-a.rate[h] * softplus_f(z));
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

// V columns c0 .. c0 + 127 of the chunk's values into [GC][128] (zeros beyond the chunk or the head's width)
__device__ __forceinline__ void gated_stage_v(const DlGatedArgs& a, const int* rows, int len, int h, int c0, float* vt) {
    const int lane = threadIdx.x & 31;
    for (int j = threadIdx.x >> 5; j < GC; j += GC_THREADS / 32) {
        const float* src = j < len ? a.v + (size_t)rows[j] * a.ldv + (size_t)h * a.vdim + c0 : nullptr;
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int cc = lane + 32 * u;
            vt[j * 128 + cc] = (src && c0 + cc < a.vdim) ? src[cc] : 0.f;
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
