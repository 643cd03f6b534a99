// Linear attention whose decay depends on the data.  Per head, state S [dim][vdim] f32, one per sequence slot:
//   channel form:  S <- diag(f_t) S + (1 - f_t) v_t^T                    f = lower + (1 - lower) sigmoid(z + bias), per channel of q
//                  S <- diag(f_t) S + k_t v_t^T                          other gates (DL_GATE_*) come with keys of their own
//   ahead form:    channel form that reads first: y_t = S_(t-1)^T q_t + (sum_d q_t bonus k_t) v_t
//   delta form:    S <- diag(f_t) S, u = sigmoid(beta_t) (v_t - S^T k_t), S <- S + k_t u^T  (its chunked kernels: delta_scan.cu)
//   head form:     S <- e^l_t S + p_t k_t v_t^T,  n <- e^l_t n + p_t k_t   one log decay l and one weight p per head and token
//   all but ahead: y_t = S_t^T q_t  (and den_t = n_t . q_t in the head form)
// Everything is f32.  A batch is any mix of sequences with one or more consecutive rows each (DlMambaBatch); a sequence
// whose first row is position 0 starts from zeros whatever its slot held.
//
// Two forms of each.  Token by token (decoding, short portions): the state in registers.  Chunked (long portions): a
// sequence's rows in chunks of GC = 64, counted from the portion's first row:
//     y_i = sum_{j <= i in chunk} ( sum_d q_i[d] D_ij[d] k_j[d] ) v_j + P^T (D_i0 q_i)       D_ij: the decay from j to i
//     P   = the state before the chunk;  state after it = D_end,0 P + sum_j (D_end,j k_j) v_j^T
// in three launches: every chunk's own sum, the prefix over a sequence's chunks (which also leaves the slot's new state),
// the outputs.  Per channel no quotient of decays is ever formed (a decay may be as small as it likes): rows are taken in
// sub-blocks of 16; between two sub-blocks the decay splits into three factors <= 1 (from the column's row to the end of its
// block, over the blocks between, from the start of the row's block to the row), inside a sub-block it is the running
// product itself.  Per head the log decays of a chunk are summed in f64.
#include "gated_common.cuh"

#define GT_TB 8                   // tokens staged per barrier pair of the token-by-token kernel
#define GT_COLS 32                // columns of S per CTA of the token-by-token kernel

// ------------------------------------------------------------------------------------------------
// token by token: a CTA owns GT_COLS columns of one head's S; thread (column, dq) keeps the rows d with (d / 4) % 4 == dq of its
// column (NR registers; rows in groups of four so that q, k and f leave shared memory as 16-byte words), the four threads
// of a column are neighbouring lanes and sum their shares of y by two shuffles.  In the head form column `vdim` is n: its
// value is 1 for every token and its output is den.  Ahead form: the bonus term is one number per token (bs).  Delta form:
// the column's share of S^T k is summed over the four lanes before the update.
// ------------------------------------------------------------------------------------------------
template <int NR, int MODE>
__global__ void __launch_bounds__(GT_COLS * 4, NR <= 32 ? 3 : 1) gated_scan_kernel(DlMambaBatch b, DlGatedArgs a) {
    constexpr int DP = NR * 4;
    constexpr bool CH = MODE != GATED_HEAD;
    extern __shared__ __align__(16) float sm[];
    const int n = blockIdx.x, h = blockIdx.y, dq = threadIdx.x & 3, c = blockIdx.z * GT_COLS + (threadIdx.x >> 2);
    const int D = a.dim, V = a.vdim, H = a.n_heads, hk = gated_k_head(a, h);
    float* qs = sm;                             // [GT_TB][DP]
    float* ks = qs + GT_TB * DP;                // [GT_TB][DP]
    float* fs = ks + GT_TB * DP;                // per channel: [GT_TB][DP]; head form: [GT_TB] decays
    float* bs = fs + GT_TB * DP;                // ahead form: [GT_TB] sums of q bonus k; delta form: [GT_TB] sigmoid(beta)
    const size_t sh = (size_t)b.seq_slot[n] * H + h;
    const bool fresh = b.seq_pos0[n] == 0, is_n = !CH && c == V, live = c < V || is_n;
    float* Sg = is_n ? a.n_state + sh * D : a.state + sh * D * V + c;       // row d at Sg[d * step]
    const size_t step = is_n ? 1 : V;
    float s[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = (i >> 2) * 16 + dq * 4 + (i & 3);
        s[i] = (live && !fresh && d < D) ? Sg[d * step] : 0.f;
    }
    const int r0 = b.seq_start[n], r1 = b.seq_start[n + 1];
    for (int rb = r0; rb < r1; rb += GT_TB) {
        const int nt = min(GT_TB, r1 - rb);
        __syncthreads();
        for (int t = threadIdx.x / 32; t < nt; t += GT_COLS * 4 / 32) {
            const size_t row = b.seq_rows[rb + t];
            const float put = CH ? 0.f : a.put[row * H + h];
            float bonus = 0.f;
            for (int d = threadIdx.x & 31; d < DP; d += 32) {
                float q = 0.f, k = 0.f, f = 0.f;
                if (d < D) {
                    q = gated_q(a, row, hk * D + d);
                    if (CH) gated_fk(a, row, h, hk, d, f, k);
                    else k = put * a.k[row * a.ldk + h * D + d];
                    if (MODE == GATED_AHEAD) bonus = fmaf(q * a.bonus[h * D + d], k, bonus);
                }
                qs[t * DP + d] = q;
                ks[t * DP + d] = k;
                if (CH) fs[t * DP + d] = f;
            }
            if (MODE == GATED_AHEAD) bonus = warp_sum(bonus);
            if ((threadIdx.x & 31) == 0) {
                if (!CH) fs[t] = expf(a.log_keep[row * H + h]);
                if (MODE == GATED_AHEAD) bs[t] = bonus;
                if (MODE == GATED_DELTA) bs[t] = sigmoid_f(a.beta[row * a.ld_beta + h]);
            }
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const size_t row = b.seq_rows[rb + t];
            float v = c < V ? a.v[row * a.ldv + h * V + c] : 1.f;
            const float keep = CH ? 0.f : fs[t];
            float y0 = 0.f, y1 = 0.f;
            if (MODE == GATED_DELTA) {          // v becomes u, the state is decayed already
                float d0 = 0.f, d1 = 0.f;
#pragma unroll
                for (int i = 0; i < NR; i += 4) {
                    const int at = t * DP + i * 4 + dq * 4;
                    const float4 k = *reinterpret_cast<const float4*>(ks + at), f = *reinterpret_cast<const float4*>(fs + at);
                    s[i] *= f.x;         d0 = fmaf(s[i], k.x, d0);
                    s[i + 1] *= f.y;     d1 = fmaf(s[i + 1], k.y, d1);
                    s[i + 2] *= f.z;     d0 = fmaf(s[i + 2], k.z, d0);
                    s[i + 3] *= f.w;     d1 = fmaf(s[i + 3], k.w, d1);
                }
                d0 += d1;
                d0 += __shfl_xor_sync(0xffffffffu, d0, 1);
                d0 += __shfl_xor_sync(0xffffffffu, d0, 2);
                v = bs[t] * (v - d0);
            }
#pragma unroll
            for (int i = 0; i < NR; i += 4) {
                const int at = t * DP + i * 4 + dq * 4;
                const float4 q = *reinterpret_cast<const float4*>(qs + at), k = *reinterpret_cast<const float4*>(ks + at);
                float4 f = make_float4(keep, keep, keep, keep);
                if (MODE == GATED_DELTA) {
                    s[i] = fmaf(k.x, v, s[i]);               y0 = fmaf(s[i], q.x, y0);
                    s[i + 1] = fmaf(k.y, v, s[i + 1]);       y1 = fmaf(s[i + 1], q.y, y1);
                    s[i + 2] = fmaf(k.z, v, s[i + 2]);       y0 = fmaf(s[i + 2], q.z, y0);
                    s[i + 3] = fmaf(k.w, v, s[i + 3]);       y1 = fmaf(s[i + 3], q.w, y1);
                    continue;
                }
                if (CH) f = *reinterpret_cast<const float4*>(fs + at);
                if (MODE == GATED_AHEAD) {
                    y0 = fmaf(s[i], q.x, y0);                s[i] = fmaf(f.x, s[i], k.x * v);
                    y1 = fmaf(s[i + 1], q.y, y1);            s[i + 1] = fmaf(f.y, s[i + 1], k.y * v);
                    y0 = fmaf(s[i + 2], q.z, y0);            s[i + 2] = fmaf(f.z, s[i + 2], k.z * v);
                    y1 = fmaf(s[i + 3], q.w, y1);            s[i + 3] = fmaf(f.w, s[i + 3], k.w * v);
                    continue;
                }
                s[i] = fmaf(f.x, s[i], k.x * v);             y0 = fmaf(s[i], q.x, y0);
                s[i + 1] = fmaf(f.y, s[i + 1], k.y * v);     y1 = fmaf(s[i + 1], q.y, y1);
                s[i + 2] = fmaf(f.z, s[i + 2], k.z * v);     y0 = fmaf(s[i + 2], q.z, y0);
                s[i + 3] = fmaf(f.w, s[i + 3], k.w * v);     y1 = fmaf(s[i + 3], q.w, y1);
            }
            float y = y0 + y1;
            y += __shfl_xor_sync(0xffffffffu, y, 1);
            y += __shfl_xor_sync(0xffffffffu, y, 2);
            if (MODE == GATED_AHEAD) y = fmaf(bs[t], v, y);
            if (live && dq == 0) {
                if (is_n) a.den[row * H + h] = y;
                else a.y[row * a.ld_y + h * V + c] = y;
            }
        }
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int d = (i >> 2) * 16 + dq * 4 + (i & 3);
            if (d < D) Sg[d * step] = s[i];
        }
    }
}

extern "C" int dl_gated_scan_supported(int dim, int vdim) { return dim >= 1 && dim <= 512 && vdim >= 1 ? 0 : -1; }

template <int NR, int MODE>
static int launch_gated_mode(const DlMambaBatch& b, int n_seq, const DlGatedArgs& a, cudaStream_t st) {
    constexpr bool CH = MODE != GATED_HEAD;
    const size_t smem = ((size_t)(CH ? 3 : 2) * GT_TB * NR * 4 + GT_TB) * sizeof(float);
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(gated_scan_kernel<NR, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) { dl_set_error("dl_gated_scan: shared memory attribute: %s", cudaGetErrorString(e)); return -(int)e; }
    }
    gated_scan_kernel<NR, MODE><<<dim3(n_seq, a.n_heads, (a.vdim + (CH ? 0 : 1) + GT_COLS - 1) / GT_COLS), GT_COLS * 4, smem, st>>>(b, a);
    return 0;
}
template <int NR>
static int launch_gated(const DlMambaBatch& b, int n_seq, const DlGatedArgs& a, cudaStream_t st) {
    if (a.f == nullptr) return launch_gated_mode<NR, GATED_HEAD>(b, n_seq, a, st);
    if (a.beta != nullptr) return launch_gated_mode<NR, GATED_DELTA>(b, n_seq, a, st);
    if (a.bonus != nullptr) return launch_gated_mode<NR, GATED_AHEAD>(b, n_seq, a, st);
    return launch_gated_mode<NR, GATED_CHANNEL>(b, n_seq, a, st);
}

extern "C" int dl_gated_scan(const DlMambaBatch* batch, int n_seq, const DlGatedArgs* args, void* stream) {
    const DlGatedArgs& a = *args;
    if (gated_args_ok(a, "dl_gated_scan")) return -1;
    if (n_seq < 1) return 0;
    cudaStream_t st = (cudaStream_t)stream;
    const int rc = a.dim <= 32 ? launch_gated<8>(*batch, n_seq, a, st) : a.dim <= 64 ? launch_gated<16>(*batch, n_seq, a, st) :
                   a.dim <= 128 ? launch_gated<32>(*batch, n_seq, a, st) : a.dim <= 256 ? launch_gated<64>(*batch, n_seq, a, st) :
                   launch_gated<128>(*batch, n_seq, a, st);
    if (rc != 0) return rc;
    LAYER_CHECK_LAUNCH("dl_gated_scan");
    return 0;
}

// ------------------------------------------------------------------------------------------------
// chunked.  Chunk c of sequence n covers rows seq_start[n] + c GC ..; its scratch slot is seq_start[n] / GC + n + c.
// Scratch: states [slots][H][D][V] | decay of the whole chunk [slots][H][D] (head form: entry 0 of D) | n sums [slots][H][D].
// ------------------------------------------------------------------------------------------------
// pass 1: a chunk's own sum of (decay to the chunk's end * k_j) v_j^T, and the decay of the whole chunk
// RT x 4 NC elements of S per thread: tiles of 16 RT rows and 64 NC columns
template <bool CH, int RT, int NC>
__global__ void __launch_bounds__(GC_THREADS) gated_chunk_state_kernel(DlMambaBatch b, DlGatedArgs a, GatedScratch sc) {
    extern __shared__ __align__(16) float sm[];
    __shared__ int rows[GC];
    __shared__ float w_s[GC];
    __shared__ double l_s[GC];
    const int n = blockIdx.x, c = blockIdx.y, h = blockIdx.z;
    int row0, len, ci;
    if (!gated_chunk_of(b, n, c, row0, len, ci)) return;
    const int D = a.dim, V = a.vdim, H = a.n_heads, D8 = (D + 7) & ~7, hk = gated_k_head(a, h);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* ks = sm;                             // [GC][D8]
    float* vt = ks + (size_t)GC * D8;           // channel form: the decays [GC][D8] first; then value tiles [GC][64 NC]
    if (threadIdx.x < GC) rows[threadIdx.x] = threadIdx.x < len ? b.seq_rows[row0 + threadIdx.x] : 0;
    if (!CH && threadIdx.x < GC) l_s[threadIdx.x] = threadIdx.x < len ? (double)a.log_keep[(size_t)b.seq_rows[row0 + threadIdx.x] * H + h] : 0.0;
    __syncthreads();
    if (!CH && threadIdx.x < GC) {              // p_j e^(l_(j+1) + ... + l_end)
        double g = 0.0;
        for (int j = threadIdx.x + 1; j < len; ++j) g += l_s[j];
        w_s[threadIdx.x] = threadIdx.x < len ? a.put[(size_t)rows[threadIdx.x] * H + h] * expf((float)g) : 0.f;
        if (threadIdx.x == 0) sc.dec[((size_t)ci * H + h) * D] = expf((float)(g + l_s[0]));
    }
    if (!CH) __syncthreads();
    if (CH) gated_stage_rows<false, false>(a, rows, len, h, hk, D8, D8, nullptr, ks, vt);
    for (int j = warp; !CH && j < GC; j += GC_THREADS / 32) {
        const size_t row = rows[j];
#pragma unroll 4
        for (int d = lane; d < D8; d += 32) ks[j * D8 + d] = j < len && d < D ? w_s[j] * a.k[row * a.ldk + h * D + d] : 0.f;
    }
    __syncthreads();
    if (CH) {
        for (int d = threadIdx.x; d < D; d += GC_THREADS) {
            float p = 1.f;
#pragma unroll 8
            for (int j = GC - 1; j >= 0; --j) {
                ks[j * D8 + d] *= p;
                p *= vt[j * D8 + d];
            }
            sc.dec[((size_t)ci * H + h) * D + d] = p;
        }
    } else {
        for (int d = threadIdx.x; d < D; d += GC_THREADS) {
            float s = 0.f;
#pragma unroll 8
            for (int j = 0; j < GC; ++j) s += ks[j * D8 + d];
            sc.ns[((size_t)ci * H + h) * D + d] = s;
        }
    }
    float* out = sc.S + ((size_t)ci * H + h) * D * V;
    const int tb = threadIdx.x >> 4, cb = threadIdx.x & 15;
    for (int c0 = 0; c0 < V; c0 += 64 * NC) {
        __syncthreads();
        gated_stage_v<64 * NC>(a, rows, len, h, c0, vt);
        __syncthreads();
        for (int d0 = 0; d0 < D; d0 += 16 * RT) {
            const int dt = d0 + tb * RT;         // this thread: RT rows of S, columns cb * 4 .. + 3 (and 64 + cb * 4 .. + 3) of the tile
            if (dt >= D8) continue;
            float acc[RT][4 * NC];
#pragma unroll
            for (int r = 0; r < RT; ++r)
#pragma unroll
                for (int u = 0; u < 4 * NC; ++u) acc[r][u] = 0.f;
#pragma unroll 2
            for (int j = 0; j < len; ++j) {
                float kk[RT], vv[4 * NC];
#pragma unroll
                for (int r = 0; r < RT; r += 4) {
                    const float4 k = *reinterpret_cast<const float4*>(ks + j * D8 + dt + r);
                    kk[r] = k.x; kk[r + 1] = k.y; kk[r + 2] = k.z; kk[r + 3] = k.w;
                }
#pragma unroll
                for (int u = 0; u < NC; ++u) {
                    const float4 v = *reinterpret_cast<const float4*>(vt + j * 64 * NC + u * 64 + cb * 4);
                    vv[4 * u] = v.x; vv[4 * u + 1] = v.y; vv[4 * u + 2] = v.z; vv[4 * u + 3] = v.w;
                }
#pragma unroll
                for (int r = 0; r < RT; ++r)
#pragma unroll
                    for (int u = 0; u < 4 * NC; ++u) acc[r][u] = fmaf(kk[r], vv[u], acc[r][u]);
            }
#pragma unroll
            for (int r = 0; r < RT; ++r)
#pragma unroll
                for (int u = 0; u < 4 * NC; ++u) {
                    const int d = dt + r, cc = c0 + (u >> 2) * 64 + cb * 4 + (u & 3);
                    if (d < D && cc < V) out[(size_t)d * V + cc] = acc[r][u];
                }
        }
    }
}

// pass 2: over a sequence's chunks in order, scratch <- the state BEFORE the chunk; the slot gets the state after the last
// one.  One thread per state element (head form: and per element of n).
template <bool CH>
__global__ void __launch_bounds__(256) gated_chunk_prefix_kernel(DlMambaBatch b, DlGatedArgs a, GatedScratch sc) {
    const int n = blockIdx.x, h = blockIdx.y;
    const int D = a.dim, V = a.vdim, H = a.n_heads, DV = D * V;
    const int e = blockIdx.z * blockDim.x + threadIdx.x;
    if (e >= DV + (CH ? 0 : D)) return;
    const bool is_n = e >= DV;
    const int s0 = b.seq_start[n], nc = (b.seq_start[n + 1] - s0 + GC - 1) / GC;
    const size_t sh = (size_t)b.seq_slot[n] * H + h, ch0 = (size_t)(s0 / GC + n) * H + h;
    float* Sg = is_n ? a.n_state + sh * D + (e - DV) : a.state + sh * DV + e;
    float R = b.seq_pos0[n] == 0 ? 0.f : *Sg;
    float* p0 = is_n ? sc.ns + ch0 * D + (e - DV) : sc.S + ch0 * DV + e;
    const size_t step = is_n ? (size_t)H * D : (size_t)H * DV, dstep = (size_t)H * D;
    const float* t0 = sc.dec + ch0 * D + (CH ? e / V : 0);
    for (int c0 = 0; c0 < nc; c0 += 8) {          // eight chunks' sums are loaded together, then chained
        float own[8], dec[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            own[i] = c0 + i < nc ? p0[(size_t)(c0 + i) * step] : 0.f;
            dec[i] = c0 + i < nc ? t0[(size_t)(c0 + i) * dstep] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (c0 + i < nc) {
                p0[(size_t)(c0 + i) * step] = R;
                R = fmaf(dec[i], R, own[i]);
            }
    }
    *Sg = R;
}

// pass 3: the outputs of a chunk.  Shared memory: Q [GC][DP] | K [GC][DP], later tiles of V and of the carried state
// [GC][64 NC] | F [GC][DP] (channel form), later the scores A [GC][GC_AS] | block decays [4][DP].
template <int MODE, int NC>
__global__ void __launch_bounds__(GC_THREADS, 2) gated_chunk_out_kernel(DlMambaBatch b, DlGatedArgs a, GatedScratch sc) {
    constexpr bool CH = MODE != GATED_HEAD;
    extern __shared__ __align__(16) float sm[];
    __shared__ int rows[GC];
    __shared__ float put_s[GC], carry_s[GC];
    __shared__ double g_s[GC];
    const int n = blockIdx.x, c = blockIdx.y, h = blockIdx.z;
    int row0, len, ci;
    if (!gated_chunk_of(b, n, c, row0, len, ci)) return;
    const int D = a.dim, V = a.vdim, H = a.n_heads, D4 = (D + 3) & ~3, DP = D4 + 4, hk = gated_k_head(a, h);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tb = threadIdx.x >> 4, cb = threadIdx.x & 15;
    float* Q = sm;
    float* K = Q + (size_t)GC * DP;
    float* F = K + max((size_t)GC * DP, (size_t)GC * 64 * NC);
    float* A = F;
    float* T = F + max(CH ? (size_t)GC * DP : 0, (size_t)GC * GC_AS);      // channel form: [4][DP]
    if (threadIdx.x < GC) {
        const int i = threadIdx.x;
        const int row = i < len ? b.seq_rows[row0 + i] : 0;
        rows[i] = row;
        if (!CH) {
            g_s[i] = i < len ? (double)a.log_keep[(size_t)row * H + h] : 0.0;
            put_s[i] = i < len ? a.put[(size_t)row * H + h] : 0.f;
        }
    }
    __syncthreads();
    if (CH) gated_stage_rows<true, false>(a, rows, len, h, hk, D4, DP, Q, K, F);
    for (int j = warp; !CH && j < GC; j += GC_THREADS / 32) {
        const size_t row = rows[j];
#pragma unroll 4
        for (int d = lane; d < D4; d += 32) {
            Q[j * DP + d] = j < len && d < D ? gated_q(a, row, h * D + d) : 0.f;
            K[j * DP + d] = j < len && d < D ? a.k[row * a.ldk + h * D + d] : 0.f;
        }
    }
    double gsum = 0.0;
    if (!CH && threadIdx.x < GC)
        for (int j = 0; j <= threadIdx.x; ++j) gsum += g_s[j];
    __syncthreads();
    if (!CH && threadIdx.x < GC) { g_s[threadIdx.x] = gsum; carry_s[threadIdx.x] = expf((float)gsum); }
    if (CH) {
        decayed_scores<MODE == GATED_AHEAD>(Q, K, F, T, D, D4, DP, MODE == GATED_AHEAD ? a.bonus + (size_t)h * D : nullptr,
                                            [&](int i, int j, float v) { A[i * GC_AS + j] = i >= j ? v : 0.f; });
    } else {
        __syncthreads();
        // A[i][j] = e^(G_i - G_j) p_j q_i . k_j, rows tb * 4 + r, columns cb + 16 u
        float acc[4][4];
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int u = 0; u < 4; ++u) acc[r][u] = 0.f;
        for (int d = 0; d < D4; d += 4) {
            float4 qv[4], kv[4];
#pragma unroll
            for (int r = 0; r < 4; ++r) qv[r] = *reinterpret_cast<const float4*>(Q + (tb * 4 + r) * DP + d);
#pragma unroll
            for (int u = 0; u < 4; ++u) kv[u] = *reinterpret_cast<const float4*>(K + (cb + 16 * u) * DP + d);
#pragma unroll
            for (int r = 0; r < 4; ++r)
#pragma unroll
                for (int u = 0; u < 4; ++u) acc[r][u] = dot4(qv[r], kv[u], acc[r][u]);
        }
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int i = tb * 4 + r, j = cb + 16 * u;
                A[i * GC_AS + j] = j <= i ? acc[r][u] * put_s[j] * expf((float)(g_s[i] - g_s[j])) : 0.f;
            }
        __syncthreads();
        // den_i = sum_j A[i][j] + e^G_i n . q_i; Q leaves scaled by e^G_i
        const float* nP = sc.ns + ((size_t)ci * H + h) * D;
        for (int i = warp; i < GC; i += GC_THREADS / 32) {
            const float cy = carry_s[i];
            float s = A[i * GC_AS + lane] + A[i * GC_AS + 32 + lane];      // zeros above the diagonal
            for (int d = lane; d < D; d += 32) {
                const float q = Q[i * DP + d] * cy;
                Q[i * DP + d] = q;
                s = fmaf(q, nP[d], s);
            }
            s = warp_sum(s);
            if (lane == 0 && i < len) a.den[(size_t)rows[i] * H + h] = s;
        }
    }
    // y = A V + Q P, V and P in tiles of 64 NC columns (P also 64 rows at a time) in the keys' place
    const float* P = sc.S + ((size_t)ci * H + h) * D * V;
    float* W = K;
    constexpr int VW = 64 * NC;
    for (int c0 = 0; c0 < V; c0 += VW) {
        const int cw = min(VW, V - c0);
        float acc[4][4 * NC];
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int u = 0; u < 4 * NC; ++u) acc[r][u] = 0.f;
        __syncthreads();
        gated_stage_v<VW>(a, rows, len, h, c0, W);
        __syncthreads();
        auto tile_mac = [&](const float* X, int ldx, int kn) {           // acc += X[rows][0 .. kn) . W[0 .. kn)[columns], kn a multiple of 4
            for (int k = 0; k < kn; k += 4) {
                float4 x[4];
#pragma unroll
                for (int r = 0; r < 4; ++r) x[r] = *reinterpret_cast<const float4*>(X + (tb * 4 + r) * ldx + k);
#pragma unroll
                for (int kk = 0; kk < 4; ++kk) {
                    float wv[4 * NC];
#pragma unroll
                    for (int u = 0; u < NC; ++u) {
                        const float4 w = *reinterpret_cast<const float4*>(W + (k + kk) * VW + u * 64 + cb * 4);
                        wv[4 * u] = w.x; wv[4 * u + 1] = w.y; wv[4 * u + 2] = w.z; wv[4 * u + 3] = w.w;
                    }
#pragma unroll
                    for (int r = 0; r < 4; ++r) {
                        const float xv = kk == 0 ? x[r].x : kk == 1 ? x[r].y : kk == 2 ? x[r].z : x[r].w;
#pragma unroll
                        for (int u = 0; u < 4 * NC; ++u) acc[r][u] = fmaf(xv, wv[u], acc[r][u]);
                    }
                }
            }
        };
        if (tb * 4 < len) tile_mac(A, GC_AS, tb * 4 + 4);
        for (int d0 = 0; d0 < D; d0 += GC) {
            const int dn = min(GC, D - d0), dn4 = (dn + 3) & ~3;
            __syncthreads();
#pragma unroll 4
            for (int d = warp; d < dn4; d += GC_THREADS / 32) {
                float p[VW / 32];
#pragma unroll
                for (int u = 0; u < VW / 32; ++u) p[u] = (d < dn && lane + 32 * u < cw) ? P[(size_t)(d0 + d) * V + c0 + lane + 32 * u] : 0.f;
#pragma unroll
                for (int u = 0; u < VW / 32; ++u) W[d * VW + lane + 32 * u] = p[u];
            }
            __syncthreads();
            if (tb * 4 < len) tile_mac(Q + d0, DP, dn4);
        }
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int i = tb * 4 + r;
            if (i >= len) continue;
            float* y = a.y + (size_t)rows[i] * a.ld_y + (size_t)h * V + c0;
#pragma unroll
            for (int u = 0; u < 4 * NC; ++u) {
                const int cc = (u >> 2) * 64 + cb * 4 + (u & 3);
                if (cc < cw) y[cc] = acc[r][u];
            }
        }
    }
}

static int gated_nc(int vdim) { return vdim <= 64 ? 1 : 2; }         // column tiles of 64 or 128
static size_t gated_state_smem(int dim, bool ch, int nc = 2) {
    const size_t D8 = (dim + 7) & ~7, vw = 64 * nc, vt = (ch && D8 > vw) ? D8 : vw;
    return (size_t)GC * (D8 + vt) * sizeof(float);
}
static size_t gated_out_smem(int dim, bool ch, int nc = 2) {
    const size_t DP = ((dim + 3) & ~3) + 4, vw = 64 * nc, k = DP > vw ? DP : vw, f = (ch && DP > GC_AS) ? DP : GC_AS;
    return ((size_t)GC * (DP + k + f) + (ch ? 4 * DP : 0)) * sizeof(float);
}

// 0 if the chunked kernels take these sizes
extern "C" int dl_gated_scan_chunked_supported(int dim, int vdim, int channel) {
    return dim >= 1 && vdim >= 1 && gated_out_smem(dim, channel) <= 225 * 1024 && gated_state_smem(dim, channel) <= 225 * 1024 ? 0 : -1;
}

// f32 of scratch for a batch of M rows in n_seq sequences
extern "C" long long dl_gated_chunk_floats(int M, int n_seq, int n_heads, int dim, int vdim) {
    return (long long)(M / GC + n_seq) * n_heads * dim * ((long long)vdim + 2);
}

template <int MODE, int NC>
static int launch_gated_out(const DlMambaBatch& b, int n_seq, int max_chunks, const DlGatedArgs& a, const GatedScratch& sc, cudaStream_t st) {
    const size_t smem = gated_out_smem(a.dim, MODE != GATED_HEAD, NC);
    cudaError_t e = cudaFuncSetAttribute(gated_chunk_out_kernel<MODE, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) { dl_set_error("gated_chunk_out: shared memory attribute: %s", cudaGetErrorString(e)); return -(int)e; }
    gated_chunk_out_kernel<MODE, NC><<<dim3(n_seq, max_chunks, a.n_heads), GC_THREADS, smem, st>>>(b, a, sc);
    return 0;
}

// pass 3 alone (the delta rule's outputs from its corrected values)
int gated_chunk_out_channel(const DlMambaBatch& b, int n_seq, int max_chunks, const DlGatedArgs& a, const GatedScratch& sc, cudaStream_t st) {
    return gated_nc(a.vdim) == 1 ? launch_gated_out<GATED_CHANNEL, 1>(b, n_seq, max_chunks, a, sc, st) : launch_gated_out<GATED_CHANNEL, 2>(b, n_seq, max_chunks, a, sc, st);
}

template <bool CH, int RT, int NC>
static int launch_gated_state(const DlMambaBatch& b, int n_seq, int max_chunks, const DlGatedArgs& a, const GatedScratch& sc, cudaStream_t st) {
    const size_t smem = gated_state_smem(a.dim, CH, NC);
    cudaError_t e = cudaFuncSetAttribute(gated_chunk_state_kernel<CH, RT, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) { dl_set_error("gated_chunk_state: shared memory attribute: %s", cudaGetErrorString(e)); return -(int)e; }
    gated_chunk_state_kernel<CH, RT, NC><<<dim3(n_seq, max_chunks, a.n_heads), GC_THREADS, smem, st>>>(b, a, sc);
    return 0;
}

template <int MODE>
static int launch_gated_chunked(const DlMambaBatch& b, int n_seq, int max_chunks, const DlGatedArgs& a, const GatedScratch& sc, cudaStream_t st) {
    constexpr bool CH = MODE != GATED_HEAD;
    const bool narrow = gated_nc(a.vdim) == 1, low = a.dim <= 64;
    int rc = narrow ? (low ? launch_gated_state<CH, 4, 1>(b, n_seq, max_chunks, a, sc, st) : launch_gated_state<CH, 8, 1>(b, n_seq, max_chunks, a, sc, st))
                    : (low ? launch_gated_state<CH, 4, 2>(b, n_seq, max_chunks, a, sc, st) : launch_gated_state<CH, 8, 2>(b, n_seq, max_chunks, a, sc, st));
    if (rc != 0) return rc;
    gated_chunk_prefix_kernel<CH><<<dim3(n_seq, a.n_heads, (a.dim * (a.vdim + (CH ? 0 : 1)) + 255) / 256), 256, 0, st>>>(b, a, sc);
    return narrow ? launch_gated_out<MODE, 1>(b, n_seq, max_chunks, a, sc, st) : launch_gated_out<MODE, 2>(b, n_seq, max_chunks, a, sc, st);
}

// max_chunks: the most chunks any sequence of the batch has; chunk_slots: M / GC + n_seq of the largest batch the scratch is for
extern "C" int dl_gated_scan_chunked(const DlMambaBatch* batch, int n_seq, int max_chunks, const DlGatedArgs* args, float* scratch,
                                     int chunk_slots, void* stream) {
    const DlGatedArgs& a = *args;
    const bool ch = a.f != nullptr;
    if (gated_args_ok(a, "dl_gated_scan_chunked")) return -1;
    if (a.beta) { dl_set_error("dl_gated_scan_chunked: the delta rule runs on dl_delta_scan_chunked"); return -1; }
    if (dl_gated_scan_chunked_supported(a.dim, a.vdim, ch) != 0 || scratch == nullptr) { dl_set_error("dl_gated_scan_chunked: sizes not supported (dim %d, vdim %d)", a.dim, a.vdim); return -1; }
    if (n_seq < 1 || max_chunks < 1) return 0;
    GatedScratch sc;
    const size_t slots = (size_t)chunk_slots;
    sc.S = scratch;
    sc.dec = sc.S + slots * a.n_heads * a.dim * a.vdim;
    sc.ns = sc.dec + slots * a.n_heads * a.dim;
    const int rc = !ch ? launch_gated_chunked<GATED_HEAD>(*batch, n_seq, max_chunks, a, sc, (cudaStream_t)stream) :
                   a.bonus ? launch_gated_chunked<GATED_AHEAD>(*batch, n_seq, max_chunks, a, sc, (cudaStream_t)stream) :
                             launch_gated_chunked<GATED_CHANNEL>(*batch, n_seq, max_chunks, a, sc, (cudaStream_t)stream);
    if (rc != 0) return rc;
    LAYER_CHECK_LAUNCH("dl_gated_scan_chunked");
    return 0;
}

// ------------------------------------------------------------------------------------------------
// gates of the matrix memory: one CTA per (sequence, head).  A token maps the running maximum u to max(b + u, a); such maps
// compose, (F, A) after (F', A') = (F + F', max(F + A', A)), so tokens are scanned in parallel: 32 by shuffles, four such
// blocks per warp, the warps' totals through shared memory (8 warps for long portions, one for short ones).
// ------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) mlstm_gates_kernel(DlMambaBatch b, DlMlstmGatesArgs a) {
    __shared__ float wF[8], wA[8];
    const int n = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5, H = a.n_heads;
    float* ug = a.u_state + (size_t)b.seq_slot[n] * H + h;
    float u = b.seq_pos0[n] == 0 ? 0.f : *ug;
    const float bi = a.bi[h], bf = a.bf[h], cap = a.cap;
    const int r0 = b.seq_start[n], r1 = b.seq_start[n + 1];
    for (int rb = r0; rb < r1; rb += nw * 128) {
        const int w0 = rb + warp * 128;
        int row[4];
        float lb[4], ai[4], F[4], A[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) { const int r = w0 + k * 32 + lane; row[k] = r < r1 ? b.seq_rows[r] : -1; }
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            ai[k] = row[k] >= 0 ? a.zi[(size_t)row[k] * a.ld + h] : 0.f;
            lb[k] = row[k] >= 0 ? a.zf[(size_t)row[k] * a.ld + h] : 0.f;
        }
        float pF = 0.f, pA = -INFINITY;                       // this warp's tokens so far, composed
        float tF[4], tA[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            tF[k] = pF; tA[k] = pA;
            F[k] = 0.f; A[k] = -INFINITY;                     // a lane without a token: the identity
            if (w0 + k * 32 < r1) {
                ai[k] = cap * tanhf((ai[k] + bi) / cap);
                lb[k] = -softplus_f(-cap * tanhf((lb[k] + bf) / cap));
                if (row[k] >= 0) { F[k] = lb[k]; A[k] = ai[k]; }
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) {
                    const float Fp = __shfl_up_sync(0xffffffffu, F[k], o), Ap = __shfl_up_sync(0xffffffffu, A[k], o);
                    if (lane >= o) { A[k] = fmaxf(F[k] + Ap, A[k]); F[k] += Fp; }
                }
                const float bF = __shfl_sync(0xffffffffu, F[k], 31), bA = __shfl_sync(0xffffffffu, A[k], 31);
                pA = fmaxf(bF + pA, bA);
                pF += bF;
            }
        }
        __syncthreads();                                      // the last round's totals have been read
        if (lane == 0) { wF[warp] = pF; wA[warp] = pA; }
        __syncthreads();
        float uw = u;                                         // u ahead of this warp's tokens, then behind the last warp's
        for (int w = 0; w < nw; ++w) {
            if (w == warp) {
                float ub = uw;
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const float us = fmaxf(tF[k] + ub, tA[k]);                        // ahead of block k
                    const float un = fmaxf(F[k] + us, A[k]);
                    float up = __shfl_up_sync(0xffffffffu, un, 1);
                    if (lane == 0) up = us;
                    if (row[k] >= 0) {
                        const size_t at = (size_t)row[k] * H + h;
                        a.log_keep[at] = lb[k] + up - un;
                        a.put[at] = expf(ai[k] - un);
                        a.floor_[at] = expf(-un);
                    }
                }
            }
            uw = fmaxf(wF[w] + uw, wA[w]);
        }
        u = uw;
    }
    if (threadIdx.x == 0) *ug = u;
}

extern "C" int dl_mlstm_gates(const DlMambaBatch* batch, int n_seq, int longest, const DlMlstmGatesArgs* args, void* stream) {
    if (args->n_heads < 1 || !(args->cap > 0.f)) { dl_set_error("dl_mlstm_gates: bad shape"); return -1; }
    if (n_seq < 1) return 0;
    mlstm_gates_kernel<<<dim3(n_seq, args->n_heads), longest > 128 ? 256 : 32, 0, (cudaStream_t)stream>>>(*batch, *args);
    LAYER_CHECK_LAUNCH("dl_mlstm_gates");
    return 0;
}

// ------------------------------------------------------------------------------------------------
// normalised heads: one warp per (row, head), half a warp for heads of up to 64 columns; four columns per lane and step (sizes and
// rows that allow it), up to 512 columns kept in registers between the sum and the scaling
// ------------------------------------------------------------------------------------------------
#define HN_WARPS 8
#define HN_CACHE 4                 // groups of four columns per lane
template <bool VEC, int LANES>
__global__ void __launch_bounds__(HN_WARPS * 32) head_norm_kernel(DlHeadNormArgs a) {
    constexpr int NC = LANES == 32 ? HN_CACHE : 1;
    const int m = blockIdx.x, lane = threadIdx.x & (LANES - 1), V = a.vdim;
    const int hh = blockIdx.y * (HN_WARPS * 32 / LANES) + threadIdx.x / LANES, h = min(hh, a.n_heads - 1);      // spare lanes repeat the last head
    if (a.xh && blockIdx.y == 0) xh_zero_tail(a.xh, a.ncap, m, a.n_heads * V, threadIdx.x, HN_WARPS * 32);
    const float* y = a.y + (size_t)m * a.ld_y + (size_t)h * V;
    const float* w = a.w + (a.w_full ? (size_t)h * V : 0);
    const float* g = a.gate ? a.gate + (size_t)m * a.ld_gate + (size_t)h * V : nullptr;
    float scale = 1.f;
    if (a.den) scale = 1.f / (fmaxf(fabsf(a.den[(size_t)m * a.n_heads + h]), a.floor_[(size_t)m * a.n_heads + h]) + 1e-6f);
    if (VEC) {
        const int n4 = V >> 2;
        float4 v[NC], gv[NC];
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < NC; ++k) {
            const int i = lane + LANES * k;
            v[k] = gv[k] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i < n4) {
                v[k] = reinterpret_cast<const float4*>(y)[i];
                if (g) gv[k] = reinterpret_cast<const float4*>(g)[i];
            }
        }
#pragma unroll
        for (int k = 0; k < NC; ++k) {
            v[k] = make_float4(v[k].x * scale, v[k].y * scale, v[k].z * scale, v[k].w * scale);
            ss = dot4(v[k], v[k], ss);
        }
#pragma unroll
        for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (hh >= a.n_heads) return;
        const float inv = 1.f / sqrtf(ss / (float)V + a.eps);
#pragma unroll
        for (int k = 0; k < NC; ++k) {
            const int i = lane + LANES * k;
            if (i >= n4) continue;
            const float4 wv = reinterpret_cast<const float4*>(w)[i];
            float4 t = make_float4(v[k].x * inv * wv.x, v[k].y * inv * wv.y, v[k].z * inv * wv.z, v[k].w * inv * wv.w);
            if (g) {
                if (a.gate_silu) { t.x *= gv[k].x; t.y *= gv[k].y; t.z *= gv[k].z; t.w *= gv[k].w; }
                t.x *= sigmoid_f(gv[k].x); t.y *= sigmoid_f(gv[k].y); t.z *= sigmoid_f(gv[k].z); t.w *= sigmoid_f(gv[k].w);
            }
            if (a.xh) {
                __nv_bfloat162 lo = __floats2bfloat162_rn(t.x, t.y), hi = __floats2bfloat162_rn(t.z, t.w);
                *reinterpret_cast<uint2*>(a.xh + xh_offset(a.ncap, m, h * V + i * 4)) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
            } else {
                reinterpret_cast<float4*>(a.out + (size_t)m * a.ld_out + (size_t)h * V)[i] = t;
            }
        }
    } else {
        if (hh >= a.n_heads) return;
        float ss = 0.f;
        for (int i = lane; i < V; i += 32) { const float t = y[i] * scale; ss = fmaf(t, t, ss); }
        const float inv = 1.f / sqrtf(warp_sum(ss) / (float)V + a.eps);
        for (int i = lane; i < V; i += 32) {
            float t = y[i] * scale * inv * w[i];
            if (g) t *= a.gate_silu ? silu_f(g[i]) : sigmoid_f(g[i]);
            if (a.xh) xh_store(a.xh, a.ncap, m, h * V + i, t);
            else a.out[(size_t)m * a.ld_out + (size_t)h * V + i] = t;
        }
    }
}

extern "C" int dl_head_norm(const DlHeadNormArgs* args, void* stream) {
    const DlHeadNormArgs& a = *args;
    if (a.M < 1 || a.n_heads < 1 || a.vdim < 1 || !a.w || (!a.out && !a.xh) || (a.den && !a.floor_)) { dl_set_error("dl_head_norm: bad arguments"); return -1; }
    const auto al = [](const void* p, long long ld) { return ((uintptr_t)p & 15) == 0 && ld % 4 == 0; };
    const bool vec = a.vdim % 4 == 0 && a.vdim <= 128 * HN_CACHE && al(a.y, a.ld_y) && al(a.w, 0) && al(a.gate, a.ld_gate) && al(a.out, a.ld_out);
    const dim3 grid(a.M, (a.n_heads + HN_WARPS - 1) / HN_WARPS);
    if (vec && a.vdim <= 64) head_norm_kernel<true, 16><<<dim3(a.M, (a.n_heads + 2 * HN_WARPS - 1) / (2 * HN_WARPS)), HN_WARPS * 32, 0, (cudaStream_t)stream>>>(a);
    else if (vec) head_norm_kernel<true, 32><<<grid, HN_WARPS * 32, 0, (cudaStream_t)stream>>>(a);
    else head_norm_kernel<false, 32><<<grid, HN_WARPS * 32, 0, (cudaStream_t)stream>>>(a);
    LAYER_CHECK_LAUNCH("dl_head_norm");
    return 0;
}
