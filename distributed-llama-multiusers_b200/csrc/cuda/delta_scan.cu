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
#define DR_WS (GC + 4)            // row strides in shared memory: W transposed, the state
#define DR_PS (DR_CB + 4)

// scratch per chunk slot and head: the states of GatedScratch, W transposed [D4][GC], and the keys decayed to the chunk's end with the chunk's
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
                for (int i = 0; i < GC; i += 4)
                    *reinterpret_cast<float4*>(W + (size_t)e * GC + i) = make_float4(Q[i * DP + e], Q[(i + 1) * DP + e], Q[(i + 2) * DP + e], Q[(i + 3) * DP + e]);
            } else {
                const int cc = e - off;
                solve_column(K + cc, 128, Nt, b_s);
                for (int i = 0; i < len; ++i) u[(size_t)rows[i] * ld_u + (size_t)h * V + c0 + cc] = K[i * 128 + cc];
            }
        }
        __syncthreads();
    }
}

// pass 2.  Shared memory: [NB][W transposed [D4][DR_WS] | keys to the end and the whole decay [GC + 1][D4 + 4]] | P [D4][DR_PS] |
// u [GC][DR_CB] | partial sums [8][GC][DR_CB].  W P: every warp takes each eighth row of P and forms all of the product (8 x 4 outputs
// per lane), the eight sums meet in shared memory.  (keys)^T u: two halves of the rows, 4 x 4 outputs per thread.
__global__ void __launch_bounds__(256) delta_chunk_walk_kernel(DlMambaBatch b, DlGatedArgs a, DeltaScratch sc, float* __restrict__ u, long long ld_u, int NB) {
    extern __shared__ __align__(16) float sm[];
    const int n = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * DR_CB, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int D = a.dim, V = a.vdim, H = a.n_heads, D4 = (D + 3) & ~3, DS = D4 + 4, stage = D4 * DR_WS + (GC + 1) * DS;
    const int s0 = b.seq_start[n], total = b.seq_start[n + 1] - s0, nc = (total + GC - 1) / GC;
    float* P = sm + (size_t)NB * stage;
    float* us = P + (size_t)D4 * DR_PS;
    float* red = us + GC * DR_CB;
    const size_t sh = (size_t)b.seq_slot[n] * H + h, ch0 = (size_t)(s0 / GC + n) * H + h;
    const bool fresh = b.seq_pos0[n] == 0;
    float* Sg = a.state + sh * D * V + c0;
    for (int e = tid; e < D4 * DR_CB; e += 256) {
        const int d = e / DR_CB, cc = e - d * DR_CB;
        P[d * DR_PS + cc] = (!fresh && d < D && c0 + cc < V) ? Sg[(size_t)d * V + cc] : 0.f;
    }
    auto issue = [&](int c, int at) {
        const size_t o = ch0 + (size_t)c * H;
        const float* w = sc.W + o * GC * D4;
        const float* ke = sc.Ke + o * (GC + 1) * D4;
        float* dw = sm + (size_t)at * stage;
        float* dk = dw + (size_t)D4 * DR_WS;
#pragma unroll 4
        for (int d = tid >> 4; d < D4; d += 16) cp_async16(dw + (size_t)d * DR_WS + (tid & 15) * 4, w + (size_t)d * GC + (tid & 15) * 4);      // half a warp per row
        for (int p = lane * 4; p < D4; p += 128)
#pragma unroll 4
            for (int i = warp; i <= GC; i += 8) cp_async16(dk + (size_t)i * DS + p, ke + (size_t)i * D4 + p);
    };
    const int ui = tid >> 2, uc = (tid & 3) * 4;               // this thread's row and four columns of u
    auto row_of = [&](int c) { return c < nc && c * GC + ui < total ? b.seq_rows[s0 + c * GC + ui] : -1; };
    auto load_own = [&](int row, float* own) {
#pragma unroll
        for (int x = 0; x < 4; ++x) own[x] = row >= 0 && c0 + uc + x < V ? u[(size_t)row * ld_u + (size_t)h * V + c0 + uc + x] : 0.f;
    };
    const int rg = lane >> 2, cg = lane & 3;                   // W P: rows rg * 8 .. + 7, columns cg * 4 .. + 3
    const int half = tid >> 7, kd = lane * 4, kc = ((tid >> 5) & 3) * 4;      // keys^T u: half of the rows, P rows kd .. + 3 (+ 128 m), columns kc .. + 3
    float own[4];
    int row = row_of(0);
    issue(0, 0);
    load_own(row, own);
    for (int c = 0; c < nc; ++c) {
        const int at = NB == 2 ? c & 1 : 0;
        const int row_next = row_of(c + 1);
        cp_async_wait_all();
        __syncthreads();                      // the chunk has landed, P is complete
        if (NB == 2 && c + 1 < nc) issue(c + 1, at ^ 1);
        const float* Wt = sm + (size_t)at * stage;
        const float* Ke = Wt + (size_t)D4 * DR_WS;
        float* Pg = sc.g.S + (ch0 + (size_t)c * H) * D * V + c0;
        for (int e = tid; e < D * DR_CB; e += 256) {           // the state ahead of this chunk
            const int d = e / DR_CB, cc = e - d * DR_CB;
            if (c0 + cc < V) Pg[(size_t)d * V + cc] = P[d * DR_PS + cc];
        }
        {
            float acc[8][4];
#pragma unroll
            for (int r = 0; r < 8; ++r) acc[r][0] = acc[r][1] = acc[r][2] = acc[r][3] = 0.f;
#pragma unroll 4
            for (int d = warp; d < D4; d += 8) {
                const float4 w0 = *reinterpret_cast<const float4*>(Wt + d * DR_WS + rg * 8), w1 = *reinterpret_cast<const float4*>(Wt + d * DR_WS + rg * 8 + 4);
                const float4 p = *reinterpret_cast<const float4*>(P + d * DR_PS + cg * 4);
                const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
                for (int r = 0; r < 8; ++r) {
                    acc[r][0] = fmaf(w[r], p.x, acc[r][0]);
                    acc[r][1] = fmaf(w[r], p.y, acc[r][1]);
                    acc[r][2] = fmaf(w[r], p.z, acc[r][2]);
                    acc[r][3] = fmaf(w[r], p.w, acc[r][3]);
                }
            }
#pragma unroll
            for (int r = 0; r < 8; ++r)
                *reinterpret_cast<float4*>(red + warp * GC * DR_CB + (rg * 8 + r) * DR_CB + cg * 4) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
        }
        __syncthreads();
        {
            float t[4] = {own[0], own[1], own[2], own[3]};
#pragma unroll
            for (int w = 0; w < 8; ++w) {
                const float4 r = *reinterpret_cast<const float4*>(red + w * GC * DR_CB + tid * 4);
                t[0] -= r.x; t[1] -= r.y; t[2] -= r.z; t[3] -= r.w;
            }
            *reinterpret_cast<float4*>(us + tid * 4) = row >= 0 ? make_float4(t[0], t[1], t[2], t[3]) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int x = 0; x < 4; ++x)
                if (row >= 0 && c0 + uc + x < V) u[(size_t)row * ld_u + (size_t)h * V + c0 + uc + x] = t[x];
            row = row_next;
            load_own(row, own);               // the next chunk's
        }
        __syncthreads();
        const float* dec = Ke + (size_t)GC * DS;
        for (int d = kd; d < D4; d += 128) {
            float acc[4][4];
#pragma unroll
            for (int r = 0; r < 4; ++r) acc[r][0] = acc[r][1] = acc[r][2] = acc[r][3] = 0.f;
#pragma unroll 8
            for (int i = half * (GC / 2); i < (half + 1) * (GC / 2); ++i) {
                const float4 k = *reinterpret_cast<const float4*>(Ke + i * DS + d), x = *reinterpret_cast<const float4*>(us + i * DR_CB + kc);
                const float kk[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    acc[r][0] = fmaf(kk[r], x.x, acc[r][0]);
                    acc[r][1] = fmaf(kk[r], x.y, acc[r][1]);
                    acc[r][2] = fmaf(kk[r], x.z, acc[r][2]);
                    acc[r][3] = fmaf(kk[r], x.w, acc[r][3]);
                }
            }
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                float4* at_p = reinterpret_cast<float4*>(P + (d + r) * DR_PS + kc);
                float4* at_r = reinterpret_cast<float4*>(red + ((d + r) * 4 + (kc >> 2)) * 4);
                if (half) {
                    *at_r = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
                } else {
                    const float4 q = *at_p;
                    const float g = dec[d + r];
                    *at_p = make_float4(fmaf(g, q.x, acc[r][0]), fmaf(g, q.y, acc[r][1]), fmaf(g, q.z, acc[r][2]), fmaf(g, q.w, acc[r][3]));
                }
            }
        }
        __syncthreads();
        for (int e = tid; e < D4 * DR_CB / 4; e += 256) {       // the second half's sums
            float4* at_p = reinterpret_cast<float4*>(P + (e >> 2) * DR_PS + (e & 3) * 4);
            const float4 q = *at_p, r = *reinterpret_cast<const float4*>(red + e * 4);
            *at_p = make_float4(q.x + r.x, q.y + r.y, q.z + r.z, q.w + r.w);
        }
        if (NB == 1 && c + 1 < nc) issue(c + 1, 0);
    }
    __syncthreads();
    for (int e = tid; e < D * DR_CB; e += 256) {
        const int d = e / DR_CB, cc = e - d * DR_CB;
        if (c0 + cc < V) Sg[(size_t)d * V + cc] = P[d * DR_PS + cc];
    }
}

#define DR_SMEM_MAX (225 * 1024)
static size_t delta_system_smem(int dim) {
    const size_t DP = ((dim + 3) & ~3) + 4, k = DP > 128 ? DP : 128, f = DP > GC_AS ? DP : GC_AS;
    return (GC * (DP + k + f) + 4 * DP) * sizeof(float);
}
static size_t delta_walk_smem(int dim, int nb) {
    const size_t D4 = (dim + 3) & ~3;
    return ((size_t)nb * (D4 * DR_WS + (GC + 1) * (D4 + 4)) + D4 * DR_PS + (size_t)9 * GC * DR_CB) * sizeof(float);
}

// 0 if the chunked kernels take these sizes
extern "C" int dl_delta_scan_chunked_supported(int dim, int vdim) {
    return dim >= 1 && vdim >= 1 && dl_gated_scan_chunked_supported(dim, vdim, 1) == 0 && delta_system_smem(dim) <= DR_SMEM_MAX && delta_walk_smem(dim, 1) <= DR_SMEM_MAX ? 0 : -1;
}

// f32 of scratch for a batch of M rows in n_seq sequences
extern "C" long long dl_delta_chunk_floats(int M, int n_seq, int n_heads, int dim, int vdim) {
    return (long long)(M / GC + n_seq) * n_heads * ((long long)dim * vdim + (2 * GC + 1) * ((dim + 3) & ~3));
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
