// The gated delta rule in chunks of GC = 64 rows of a sequence (token by token: gated_scan.cu).  Per head, with decays f per key
// channel, D_ij the decay from row j to row i, P the state ahead of the chunk, b_i = sigmoid(beta_i):
//     u_i = b_i ( v_i - sum_{j < i} (k_i . D_ij k_j) u_j - P^T (D_i0 k_i) )
//     y_i = sum_{j <= i} (q_i . D_ij k_j) u_j + P^T (D_i0 q_i),      state after the chunk: D_end,0 P + sum_j (D_end,j k_j) u_j^T
// The u_i of a chunk are the solution of a unit lower triangular system whose right side is linear in P, so in three launches:
//     1  every chunk by itself:  N_ij = b_i k_i . D_ij k_j;  (I + N) W = b D_.0 k,  (I + N) U = b v;  also the keys decayed to the
//        chunk's end and the chunk's whole decay                                               (u_i = U_i - P^T W_i)
//     2  a sequence's chunks in order, P in shared memory, 16 columns of it per CTA:  u = U - W P,  P <- D_end,0 P + (D_end,j k_j)^T u;
//        every chunk's P is left for
//     3  the outputs: gated_chunk_out_kernel of gated_scan.cu with u in the values' place
// All f32; no quotient of decays is ever formed (decayed_scores()).  Rows a sequence does not have get k = 0, b = 0.
#include "gated_common.cuh"
#include "mma_common.cuh"

#define DR_CB 16                  // columns of the state per CTA of the walk
#define DR_ROWS (2 * GC + 1)      // staged rows per chunk of the walk

// scratch per chunk slot and head: the states of GatedScratch, W [GC][D4], and the keys decayed to the chunk's end with the chunk's
// whole decay as one more row, Ke [GC + 1][D4]
struct DeltaScratch { GatedScratch g; float* W; float* Ke; };

// one column of (I + N) X = b R by substitution, in place: x[i * ld], i < GC; Nt [GC][GC_AS] holds N transposed.  Rows in blocks of
// 16: the rows ahead of a block are read back, the block itself stays in registers.
__device__ __forceinline__ void solve_column(float* x, int ld, const float* Nt, const float* b_s) {
#pragma unroll 1
    for (int i0 = 0; i0 < GC; i0 += 16) {
        float r[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) r[i] = b_s[i0 + i] * x[(size_t)(i0 + i) * ld];
#pragma unroll 4
        for (int j = 0; j < i0; ++j) {
            const float xj = x[(size_t)j * ld];
            const float* nt = Nt + j * GC_AS + i0;
#pragma unroll
            for (int i = 0; i < 16; i += 4) {
                const float4 n = *reinterpret_cast<const float4*>(nt + i);
                r[i] = fmaf(-n.x, xj, r[i]);
                r[i + 1] = fmaf(-n.y, xj, r[i + 1]);
                r[i + 2] = fmaf(-n.z, xj, r[i + 2]);
                r[i + 3] = fmaf(-n.w, xj, r[i + 3]);
            }
        }
#pragma unroll
        for (int j = 0; j < 15; ++j) {
            const float* nt = Nt + (i0 + j) * GC_AS + i0;
#pragma unroll
            for (int i = 0; i < 16; ++i)
                if (i > j) r[i] = fmaf(-nt[i], r[j], r[i]);
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) x[(size_t)(i0 + i) * ld] = r[i];
    }
}

// pass 1.  Shared memory: Q, the keys as rows (later W) [GC][DP] | K, the keys as columns [GC][DP], later values [GC][128] | F, the
// decays [GC][DP], later N transposed [GC][GC_AS] | block decays [4][DP].
__global__ void __launch_bounds__(GC_THREADS, 2) delta_chunk_system_kernel(DlMambaBatch b, DlGatedArgs a, DeltaScratch sc, float* __restrict__ u, long long ld_u) {
    extern __shared__ __align__(16) float sm[];
    __shared__ int rows[GC];
    __shared__ float b_s[GC];
    const int n = blockIdx.x, c = blockIdx.y, h = blockIdx.z;
    int row0, len, ci;
    if (!gated_chunk_of(b, n, c, row0, len, ci)) return;
    const int D = a.dim, V = a.vdim, H = a.n_heads, D4 = (D + 3) & ~3, DP = D4 + 4, hk = gated_k_head(a, h);
    float* Q = sm;
    float* K = Q + (size_t)GC * DP;
    float* F = K + max((size_t)GC * DP, (size_t)GC * 128);
    float* T = F + max((size_t)GC * DP, (size_t)GC * GC_AS);
    if (threadIdx.x < GC) {
        const int i = threadIdx.x, row = i < len ? b.seq_rows[row0 + i] : 0;
        rows[i] = row;
        b_s[i] = i < len ? sigmoid_f(a.beta[(size_t)row * a.ld_beta + h]) : 0.f;
    }
    __syncthreads();
    gated_stage_rows<false, true>(a, rows, len, h, hk, D4, DP, Q, K, F);
    __syncthreads();
    float* Nt = F;
    decayed_scores<false>(Q, K, F, T, D, D4, DP, nullptr, [&](int i, int j, float v) { if (i > j) Nt[j * GC_AS + i] = b_s[i] * v; });
    float* Ke = sc.Ke + ((size_t)ci * H + h) * (GC + 1) * D4;
    for (int t = threadIdx.x; t < 4 * D4; t += GC_THREADS) {
        const int bk = t / D4, d = t - bk * D4;
        float p = 1.f;
        for (int v = bk + 1; v < 4; ++v) p *= T[v * DP + d];
#pragma unroll
        for (int i = 0; i < 16; ++i) Ke[(size_t)(bk * 16 + i) * D4 + d] = K[(bk * 16 + i) * DP + d] * p;
        if (bk == 0) Ke[(size_t)GC * D4 + d] = p * T[d];
    }
    __syncthreads();
    float* W = sc.W + ((size_t)ci * H + h) * GC * D4;
    for (int c0 = 0; c0 < V; c0 += 128) {
        const int cw = min(128, V - c0), off = c0 == 0 ? D4 : 0;      // the first round also solves for W
        gated_stage_v<128>(a, rows, len, h, c0, K);
        __syncthreads();
        for (int e = threadIdx.x; e < off + cw; e += GC_THREADS) {
            if (e < off) {
                solve_column(Q + e, DP, Nt, b_s);
                for (int i = 0; i < GC; ++i) W[(size_t)i * D4 + e] = Q[i * DP + e];
            } else {
                const int cc = e - off;
                solve_column(K + cc, 128, Nt, b_s);
                for (int i = 0; i < len; ++i) u[(size_t)rows[i] * ld_u + (size_t)h * V + c0 + cc] = K[i * 128 + cc];
            }
        }
        __syncthreads();
    }
}

// pass 2.  Shared memory: [NB][W [GC] | keys to the end, whole decay [GC + 1]][D4 + 4] | P [D4][DR_CB] | u [GC][DR_CB].
__global__ void __launch_bounds__(256) delta_chunk_walk_kernel(DlMambaBatch b, DlGatedArgs a, DeltaScratch sc, float* __restrict__ u, long long ld_u, int NB) {
    extern __shared__ __align__(16) float sm[];
    const int n = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * DR_CB, tid = threadIdx.x;
    const int D = a.dim, V = a.vdim, H = a.n_heads, D4 = (D + 3) & ~3, DS = D4 + 4;
    const int s0 = b.seq_start[n], total = b.seq_start[n + 1] - s0, nc = (total + GC - 1) / GC;
    float* buf = sm;
    float* P = buf + (size_t)NB * DR_ROWS * DS;
    float* us = P + (size_t)D4 * DR_CB;
    const size_t sh = (size_t)b.seq_slot[n] * H + h, ch0 = (size_t)(s0 / GC + n) * H + h;
    const bool fresh = b.seq_pos0[n] == 0;
    float* Sg = a.state + sh * D * V + c0;
    for (int e = tid; e < D4 * DR_CB; e += 256) {
        const int d = e / DR_CB, cc = e - d * DR_CB;
        P[e] = (!fresh && d < D && c0 + cc < V) ? Sg[(size_t)d * V + cc] : 0.f;
    }
    auto issue = [&](int c, int at) {         // a warp per row
        const size_t o = ch0 + (size_t)c * H;
        const float* w = sc.W + o * GC * D4;
        const float* ke = sc.Ke + o * (GC + 1) * D4 - (size_t)GC * D4;
        float* dst = buf + (size_t)at * DR_ROWS * DS;
        for (int p = (tid & 31) * 4; p < D4; p += 128)
#pragma unroll 4
            for (int i = tid >> 5; i < DR_ROWS; i += 8) cp_async16(dst + (size_t)i * DS + p, (i < GC ? w : ke) + (size_t)i * D4 + p);
    };
    const int ui = tid >> 2, uc = (tid & 3) * 4;               // step A: this thread's row and four columns of u
    const int half = tid >> 7, cols = DR_CB / 2;               // step B: half of the columns of rows d = tid % 128 + 128 x of P
    issue(0, 0);
    for (int c = 0; c < nc; ++c) {
        const int at = NB == 2 ? c & 1 : 0, len = min(GC, total - c * GC);
        float own[4] = {0.f, 0.f, 0.f, 0.f};
        float* ug = nullptr;
        if (ui < len) {
            ug = u + (size_t)b.seq_rows[s0 + c * GC + ui] * ld_u + (size_t)h * V + c0 + uc;
#pragma unroll
            for (int x = 0; x < 4; ++x)
                if (c0 + uc + x < V) own[x] = ug[x];
        }
        cp_async_wait_all();
        __syncthreads();                      // the chunk has landed, P is complete
        if (NB == 2 && c + 1 < nc) issue(c + 1, at ^ 1);
        const float* W = buf + (size_t)at * DR_ROWS * DS;
        const float* Ke = W + (size_t)GC * DS;
        float* Pg = sc.g.S + (ch0 + (size_t)c * H) * D * V + c0;
        for (int e = tid; e < D * DR_CB; e += 256) {           // the state ahead of this chunk
            const int d = e / DR_CB, cc = e - d * DR_CB;
            if (c0 + cc < V) Pg[(size_t)d * V + cc] = P[e];
        }
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
        for (int d = 0; d < D4; d += 4) {
            const float4 w = *reinterpret_cast<const float4*>(W + ui * DS + d);
            const float wv[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float4 p = *reinterpret_cast<const float4*>(P + (d + x) * DR_CB + uc);
                acc[0] = fmaf(wv[x], p.x, acc[0]);
                acc[1] = fmaf(wv[x], p.y, acc[1]);
                acc[2] = fmaf(wv[x], p.z, acc[2]);
                acc[3] = fmaf(wv[x], p.w, acc[3]);
            }
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const float t = own[x] - acc[x];
            us[ui * DR_CB + uc + x] = ui < len ? t : 0.f;
            if (ug && c0 + uc + x < V) ug[x] = t;
        }
        __syncthreads();
        const float* dec = Ke + (size_t)GC * DS;
        for (int d = tid & 127; d < D; d += 128) {
            float p[8];
            const float g = dec[d];
#pragma unroll
            for (int x = 0; x < 8; ++x) p[x] = g * P[d * DR_CB + half * cols + x];
#pragma unroll 8
            for (int i = 0; i < GC; ++i) {
                const float k = Ke[i * DS + d];
                const float4 u0 = *reinterpret_cast<const float4*>(us + i * DR_CB + half * cols), u1 = *reinterpret_cast<const float4*>(us + i * DR_CB + half * cols + 4);
                p[0] = fmaf(k, u0.x, p[0]); p[1] = fmaf(k, u0.y, p[1]); p[2] = fmaf(k, u0.z, p[2]); p[3] = fmaf(k, u0.w, p[3]);
                p[4] = fmaf(k, u1.x, p[4]); p[5] = fmaf(k, u1.y, p[5]); p[6] = fmaf(k, u1.z, p[6]); p[7] = fmaf(k, u1.w, p[7]);
            }
#pragma unroll
            for (int x = 0; x < 8; ++x) P[d * DR_CB + half * cols + x] = p[x];
        }
        if (NB == 1 && c + 1 < nc) {
            __syncthreads();
            issue(c + 1, 0);
        }
    }
    __syncthreads();
    for (int e = tid; e < D * DR_CB; e += 256) {
        const int d = e / DR_CB, cc = e - d * DR_CB;
        if (c0 + cc < V) Sg[(size_t)d * V + cc] = P[e];
    }
}

#define DR_SMEM_MAX (225 * 1024)
static size_t delta_system_smem(int dim) {
    const size_t DP = ((dim + 3) & ~3) + 4, k = DP > 128 ? DP : 128, f = DP > GC_AS ? DP : GC_AS;
    return (GC * (DP + k + f) + 4 * DP) * sizeof(float);
}
static size_t delta_walk_smem(int dim, int nb) {
    const size_t D4 = (dim + 3) & ~3;
    return ((size_t)nb * DR_ROWS * (D4 + 4) + D4 * DR_CB + (size_t)GC * DR_CB) * sizeof(float);
}

// 0 if the chunked kernels take these sizes
extern "C" int dl_delta_scan_chunked_supported(int dim, int vdim) {
    return dim >= 1 && vdim >= 1 && dl_gated_scan_chunked_supported(dim, vdim, 1) == 0 && delta_system_smem(dim) <= DR_SMEM_MAX && delta_walk_smem(dim, 1) <= DR_SMEM_MAX ? 0 : -1;
}

// f32 of scratch for a batch of M rows in n_seq sequences
extern "C" long long dl_delta_chunk_floats(int M, int n_seq, int n_heads, int dim, int vdim) {
    return (long long)(M / GC + n_seq) * n_heads * ((long long)dim * vdim + DR_ROWS * ((dim + 3) & ~3));
}

extern "C" int dl_delta_scan_chunked(const DlMambaBatch* batch, int n_seq, int max_chunks, const DlGatedArgs* args, float* scratch,
                                     int chunk_slots, float* u, long long ld_u, void* stream) {
    DlGatedArgs a = *args;
    if (gated_args_ok(a, "dl_delta_scan_chunked")) return -1;
    if (!a.beta || !a.f || a.gate == DL_GATE_LOWER || scratch == nullptr || u == nullptr || dl_delta_scan_chunked_supported(a.dim, a.vdim) != 0) {
        dl_set_error("dl_delta_scan_chunked: bad arguments (dim %d, vdim %d)", a.dim, a.vdim);
        return -1;
    }
    if (n_seq < 1 || max_chunks < 1) return 0;
    cudaStream_t st = (cudaStream_t)stream;
    const size_t slots = (size_t)chunk_slots * a.n_heads, D4 = (a.dim + 3) & ~3;
    DeltaScratch sc;                          // the copied arrays first: they start on 16 bytes
    sc.W = scratch;
    sc.Ke = sc.W + slots * GC * D4;
    sc.g.S = sc.Ke + slots * (GC + 1) * D4;
    sc.g.dec = sc.g.ns = nullptr;
    const int nb = delta_walk_smem(a.dim, 2) <= DR_SMEM_MAX ? 2 : 1;
    const size_t smem1 = delta_system_smem(a.dim), smem2 = delta_walk_smem(a.dim, nb);
    cudaError_t e = cudaFuncSetAttribute(delta_chunk_system_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_chunk_walk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem2);
    if (e != cudaSuccess) { dl_set_error("dl_delta_scan_chunked: shared memory attribute: %s", cudaGetErrorString(e)); return -(int)e; }
    delta_chunk_system_kernel<<<dim3(n_seq, max_chunks, a.n_heads), GC_THREADS, smem1, st>>>(*batch, a, sc, u, ld_u);
    delta_chunk_walk_kernel<<<dim3(n_seq, a.n_heads, (a.vdim + DR_CB - 1) / DR_CB), 256, smem2, st>>>(*batch, a, sc, u, ld_u, nb);
    a.v = u;
    a.ldv = ld_u;
    a.beta = nullptr;
    const int rc = gated_chunk_out_channel(*batch, n_seq, max_chunks, a, sc.g, st);
    if (rc != 0) return rc;
    LAYER_CHECK_LAUNCH("dl_delta_scan_chunked");
    return 0;
}
