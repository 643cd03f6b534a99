// Selective scan with a state per channel (Mamba): per channel c and state index n, all f32,
//     step  = softplus(dt_c + dt_bias_c)                       S[c][n] <- exp(-step exp(A_log[c][n])) S[c][n] + step x_c B_n
//     y_c   = sum_n S[c][n] C_n + D_c x_c                      out_c = y_c * silu(z_c)
// (A2 = -exp(A_log) / ln 2: the decay is 2^(step A2)).  A batch is any mix of sequences with one or more consecutive rows each; a
// sequence whose first row is position 0 starts from zeros whatever its slot held.
//
// Three forms.
//   * One row per sequence (decoding): four lanes share a channel, everything a row needs is loaded at once.
//   * Short portions (and more than 32 state entries): a CTA owns SS_CH channels of one sequence, four neighbouring lanes share
//     a channel and keep its state in registers (lane l holds the n with (n / 4) % 4 == l, so that B and C leave shared memory as
//     16-byte words); SS_TB tokens are staged per barrier pair, the next tile's loads in flight while a tile is walked.
//   * Long portions: chunks of SC rows of a sequence in parallel, thread = channel with the whole state in registers (a warp reads
//     32 neighbouring channels of a row; B and C of the chunk sit in shared memory).  A chunk's decay is 2^(A2 * sum of its
//     steps), so the first launch leaves every chunk's own state from zeros and its sum of steps, the second runs the prefix over a
//     sequence's chunks (state before each chunk; the slot's new state), the third walks every chunk again from its state.
#include "layer_common.cuh"
#include "../../../include/dllama_b200.h"

#define SS_CH 32
#define SS_TB 16
#define SS_THREADS (SS_CH * 4)
#define SC DL_SELECTIVE_CHUNK
#define SC_THREADS 128

__device__ __forceinline__ float ss_ex2(float x) {            // arguments <= 0: flushing tiny decays to zero is exact enough
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// ------------------------------------------------------------------------------------------------
// one row per sequence: thread (channel, quarter of the state), NS state entries each
// ------------------------------------------------------------------------------------------------
template <int NS>
__global__ void __launch_bounds__(SS_THREADS) selective_step_kernel(DlMambaBatch b, DlSelectiveArgs a) {
    const int n = blockIdx.x, l = threadIdx.x & 3, ch = blockIdx.y * SS_CH + (threadIdx.x >> 2), N = a.state, inner = a.inner;
    const bool live = ch < inner;
    const size_t row = b.seq_rows[b.seq_start[n]];
    float* Sg = a.state_pool + ((size_t)b.seq_slot[n] * inner + ch) * N;
    const bool fresh = b.seq_pos0[n] == 0;
    float s[NS], A[NS], B[NS], C[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int k = (i >> 2) * 16 + l * 4 + (i & 3);
        const bool in = live && k < N;
        s[i] = (in && !fresh) ? Sg[k] : 0.f;
        A[i] = in ? a.A2[(size_t)ch * N + k] : 0.f;
        B[i] = in ? a.B[row * a.ld_bc + k] : 0.f;
        C[i] = in ? a.C[row * a.ld_bc + k] : 0.f;
    }
    const float x = live ? a.x[row * a.ld_x + ch] : 0.f, z = live && a.z ? a.z[row * a.ld_z + ch] : 0.f, Dc = live ? a.D[ch] : 0.f;
    const float dt = live ? softplus_f(a.dt[row * a.ld_dt + ch] + a.dt_bias[ch]) : 0.f, dx = dt * x;
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        s[i] = fmaf(ss_ex2(dt * A[i]), s[i], dx * B[i]);
        y = fmaf(s[i], C[i], y);
    }
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int k = (i >> 2) * 16 + l * 4 + (i & 3);
        if (live && k < N) Sg[k] = s[i];
    }
    y += __shfl_xor_sync(0xffffffffu, y, 1);
    y += __shfl_xor_sync(0xffffffffu, y, 2);
    y = fmaf(Dc, x, y);
    if (a.z) y *= silu_f(z);
    if (l == 0 && live) {
        if (a.xh) xh_store(a.xh, a.ncap, (int)row, ch, y);
        else a.y[row * a.ld_y + ch] = y;
    }
    if (a.xh && blockIdx.y == gridDim.y - 1) xh_zero_tail(a.xh, a.ncap, (int)row, inner, threadIdx.x, SS_THREADS);
}

// ------------------------------------------------------------------------------------------------
// short portions
// ------------------------------------------------------------------------------------------------
template <int NS>            // state indices per lane: state <= 4 * NS
__global__ void __launch_bounds__(SS_THREADS) selective_scan_kernel(DlMambaBatch b, DlSelectiveArgs a) {
    constexpr int NP = 4 * NS, RX = SS_TB * SS_CH / SS_THREADS, RB = SS_TB * NP / SS_THREADS;
    __shared__ __align__(16) float B_s[SS_TB][NP], C_s[SS_TB][NP];
    __shared__ float dt_s[SS_TB][SS_CH], x_s[SS_TB][SS_CH], y_s[SS_TB][SS_CH + 1];
    __shared__ int row_s[2][SS_TB];
    const int n = blockIdx.x, ch0 = blockIdx.y * SS_CH, tid = threadIdx.x, lc = tid >> 2, l = tid & 3, ch = ch0 + lc;
    const int N = a.state, inner = a.inner;
    const bool live = ch < inner, fresh = b.seq_pos0[n] == 0;
    float* Sg = a.state_pool + ((size_t)b.seq_slot[n] * inner + ch) * N;
    float s[NS], A[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int k = (i >> 2) * 16 + l * 4 + (i & 3);
        const bool in = live && k < N;
        s[i] = (in && !fresh) ? Sg[k] : 0.f;
        A[i] = in ? a.A2[(size_t)ch * N + k] : 0.f;
    }
    const float Dc = live ? a.D[ch] : 0.f;
    // staging roles: element u of this thread is (token u * 4 + warp, channel lane) and entry (u * SS_THREADS + tid) of B and C
    const int warp = tid >> 5, lane = tid & 31, lch = ch0 + lane;
    const float bias = lch < inner ? a.dt_bias[lch] : 0.f;
    const int r0 = b.seq_start[n], r1 = b.seq_start[n + 1];
    float px[RX], pdt[RX], pB[RB], pC[RB];
    auto fetch = [&](int buf) {                  // row_s[buf] holds the tile's rows (-1: none)
#pragma unroll
        for (int u = 0; u < RX; ++u) {
            const int row = row_s[buf][u * 4 + warp];
            const bool in = row >= 0 && lch < inner;
            px[u] = in ? a.x[(size_t)row * a.ld_x + lch] : 0.f;
            pdt[u] = in ? a.dt[(size_t)row * a.ld_dt + lch] + bias : 0.f;
        }
#pragma unroll
        for (int u = 0; u < RB; ++u) {
            const int e = u * SS_THREADS + tid, k = e % NP, row = row_s[buf][e / NP];
            const bool in = row >= 0 && k < N;
            pB[u] = in ? a.B[(size_t)row * a.ld_bc + k] : 0.f;
            pC[u] = in ? a.C[(size_t)row * a.ld_bc + k] : 0.f;
        }
    };
    if (tid < SS_TB) row_s[0][tid] = r0 + tid < r1 ? b.seq_rows[r0 + tid] : -1;
    __syncthreads();
    fetch(0);
    int buf = 0;
    for (int rb = r0; rb < r1; rb += SS_TB, buf ^= 1) {
        const int nt = min(SS_TB, r1 - rb);
#pragma unroll
        for (int u = 0; u < RX; ++u) {
            x_s[u * 4 + warp][lane] = px[u];
            dt_s[u * 4 + warp][lane] = softplus_f(pdt[u]);
        }
#pragma unroll
        for (int u = 0; u < RB; ++u) {
            const int e = u * SS_THREADS + tid;
            B_s[e / NP][e % NP] = pB[u];
            C_s[e / NP][e % NP] = pC[u];
        }
        if (tid < SS_TB) row_s[buf ^ 1][tid] = rb + SS_TB + tid < r1 ? b.seq_rows[rb + SS_TB + tid] : -1;
        __syncthreads();
        if (rb + SS_TB < r1) fetch(buf ^ 1);
#pragma unroll 2
        for (int t = 0; t < nt; ++t) {
            const float dt = dt_s[t][lc], x = x_s[t][lc], dx = dt * x;
            float y0 = 0.f, y1 = 0.f;
#pragma unroll
            for (int i = 0; i < NS; i += 4) {
                const float4 B = *reinterpret_cast<const float4*>(&B_s[t][i * 4 + l * 4]), C = *reinterpret_cast<const float4*>(&C_s[t][i * 4 + l * 4]);
                s[i] = fmaf(ss_ex2(dt * A[i]), s[i], dx * B.x);              y0 = fmaf(s[i], C.x, y0);
                s[i + 1] = fmaf(ss_ex2(dt * A[i + 1]), s[i + 1], dx * B.y);  y1 = fmaf(s[i + 1], C.y, y1);
                s[i + 2] = fmaf(ss_ex2(dt * A[i + 2]), s[i + 2], dx * B.z);  y0 = fmaf(s[i + 2], C.z, y0);
                s[i + 3] = fmaf(ss_ex2(dt * A[i + 3]), s[i + 3], dx * B.w);  y1 = fmaf(s[i + 3], C.w, y1);
            }
            float y = y0 + y1;
            y += __shfl_xor_sync(0xffffffffu, y, 1);
            y += __shfl_xor_sync(0xffffffffu, y, 2);
            if (l == 0) y_s[t][lc] = fmaf(Dc, x, y);
        }
        __syncthreads();
        if (lch < inner) {                       // the tile's outputs: (token, channel) per thread
#pragma unroll
            for (int u = 0; u < RX; ++u) {
                const int t = u * 4 + warp;
                if (t >= nt) break;
                const int row = row_s[buf][t];
                float v = y_s[t][lane];
                if (a.z) v *= silu_f(a.z[(size_t)row * a.ld_z + lch]);
                if (a.xh) xh_store(a.xh, a.ncap, row, lch, v);
                else a.y[(size_t)row * a.ld_y + lch] = v;
            }
        }
        if (a.xh && blockIdx.y == gridDim.y - 1)
            for (int t = 0; t < nt; ++t) xh_zero_tail(a.xh, a.ncap, row_s[buf][t], inner, tid, SS_THREADS);
        __syncthreads();
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < NS; ++i) {
            const int k = (i >> 2) * 16 + l * 4 + (i & 3);
            if (k < N) Sg[k] = s[i];
        }
    }
}

extern "C" int dl_selective_scan_supported(int state) { return state >= 1 && state <= 128 ? 0 : -1; }

static int selective_args_ok(const DlSelectiveArgs& a, const char* who) {
    if (a.inner < 1 || dl_selective_scan_supported(a.state) != 0 || (!a.y && !a.xh)) { dl_set_error("%s: bad shape (inner %d, state %d)", who, a.inner, a.state); return -1; }
    return 0;
}

extern "C" int dl_selective_scan(const DlMambaBatch* batch, int n_seq, int longest, const DlSelectiveArgs* args, void* stream) {
    const DlSelectiveArgs& a = *args;
    if (selective_args_ok(a, "dl_selective_scan")) return -1;
    if (n_seq < 1) return 0;
    cudaStream_t st = (cudaStream_t)stream;
    const dim3 grid(n_seq, (a.inner + SS_CH - 1) / SS_CH);
#define SS_CASE(NS_)                                                                                  \
    do {                                                                                              \
        if (longest <= 1) selective_step_kernel<NS_><<<grid, SS_THREADS, 0, st>>>(*batch, a);         \
        else selective_scan_kernel<NS_><<<grid, SS_THREADS, 0, st>>>(*batch, a);                      \
    } while (0)
    if (a.state <= 16) SS_CASE(4);
    else if (a.state <= 32) SS_CASE(8);
    else if (a.state <= 64) SS_CASE(16);
    else SS_CASE(32);
#undef SS_CASE
    LAYER_CHECK_LAUNCH("dl_selective_scan");
    return 0;
}

// ------------------------------------------------------------------------------------------------
// chunked.  Chunk c of sequence n covers rows seq_start[n] + c SC ..; its scratch slot is seq_start[n] / SC + n + c.  Scratch:
// states [slots][state][inner] (channels contiguous) | sums of steps [slots][inner].
// ------------------------------------------------------------------------------------------------
// passes 1 and 3: grid (sequence, chunk, SC_THREADS channels); thread = channel.  OUT: from the state before the chunk, with outputs
template <int N, bool OUT>
__global__ void __launch_bounds__(SC_THREADS) selective_chunk_kernel(DlMambaBatch b, DlSelectiveArgs a, float* __restrict__ states, float* __restrict__ sums) {
    __shared__ __align__(16) float B_s[SC][N], C_s[OUT ? SC : 1][N];
    __shared__ int row_s[SC];
    const int n = blockIdx.x, c = blockIdx.y, tid = threadIdx.x, ch = blockIdx.z * SC_THREADS + tid;
    const int s0 = b.seq_start[n], total = b.seq_start[n + 1] - s0;
    if (c * SC >= total) return;
    const int len = min(SC, total - c * SC), row0 = s0 + c * SC, inner = a.inner;
    const size_t ci = s0 / SC + n + c;
    if (tid < SC) row_s[tid] = tid < len ? b.seq_rows[row0 + tid] : -1;
    __syncthreads();
    for (int e = tid; e < SC * N; e += SC_THREADS) {
        const int t = e / N, k = e % N, row = row_s[t];
        const bool in = row >= 0 && k < a.state;
        B_s[t][k] = in ? a.B[(size_t)row * a.ld_bc + k] : 0.f;
        if (OUT) C_s[t][k] = in ? a.C[(size_t)row * a.ld_bc + k] : 0.f;
    }
    const bool live = ch < inner;
    const int cc = live ? ch : inner - 1;                     // an idle thread walks the last channel and stores nothing
    float s[N], A[N];
#pragma unroll
    for (int k = 0; k < N; ++k) {
        A[k] = k < a.state ? a.A2[(size_t)cc * a.state + k] : 0.f;
        s[k] = OUT && k < a.state ? states[(ci * a.state + k) * inner + cc] : 0.f;
    }
    const float bias = a.dt_bias[cc], Dc = a.D[cc];
    __syncthreads();
    float sum = 0.f;
    constexpr int PF = 4;                                     // tokens whose loads are in flight
    float px[PF], pdt[PF], pz[PF];
    auto fetch = [&](int t, float& x, float& dt, float& z) {
        const size_t row = t < len ? row_s[t] : row_s[0];
        x = a.x[row * a.ld_x + cc];
        dt = a.dt[row * a.ld_dt + cc];
        z = OUT && a.z ? a.z[row * a.ld_z + cc] : 0.f;
    };
#pragma unroll
    for (int u = 0; u < PF; ++u) fetch(u, px[u], pdt[u], pz[u]);
    for (int t0 = 0; t0 < len; t0 += PF) {
#pragma unroll
        for (int u = 0; u < PF; ++u) {
            const int t = t0 + u;
            const float x = px[u], dtr = pdt[u], z = pz[u];
            fetch(t + PF, px[u], pdt[u], pz[u]);
            if (t < len) {
                const float dt = softplus_f(dtr + bias), dx = dt * x;
                float y0 = 0.f, y1 = 0.f;
                if (!OUT) sum += dt;
#pragma unroll
                for (int k = 0; k < N; k += 4) {
                    const float4 B = *reinterpret_cast<const float4*>(&B_s[t][k]);
                    s[k] = fmaf(ss_ex2(dt * A[k]), s[k], dx * B.x);
                    s[k + 1] = fmaf(ss_ex2(dt * A[k + 1]), s[k + 1], dx * B.y);
                    s[k + 2] = fmaf(ss_ex2(dt * A[k + 2]), s[k + 2], dx * B.z);
                    s[k + 3] = fmaf(ss_ex2(dt * A[k + 3]), s[k + 3], dx * B.w);
                    if (OUT) {
                        const float4 C = *reinterpret_cast<const float4*>(&C_s[t][k]);
                        y0 = fmaf(s[k], C.x, y0);
                        y1 = fmaf(s[k + 1], C.y, y1);
                        y0 = fmaf(s[k + 2], C.z, y0);
                        y1 = fmaf(s[k + 3], C.w, y1);
                    }
                }
                if (OUT) {
                    float y = fmaf(Dc, x, y0 + y1);
                    if (a.z) y *= z * __fdividef(1.f, 1.f + expf(-z));
                    const int row = row_s[t];
                    if (a.xh) {                               // neighbouring lanes hold neighbouring channels: pairs leave as 4 bytes
                        const float y_next = __shfl_down_sync(0xffffffffu, live ? y : 0.f, 1);
                        if (live && !(tid & 1)) {
                            __nv_bfloat162 p = __floats2bfloat162_rn(y, y_next);
                            *reinterpret_cast<uint32_t*>(a.xh + xh_offset(a.ncap, row, ch)) = *reinterpret_cast<uint32_t*>(&p);
                        }
                    } else if (live) {
                        a.y[(size_t)row * a.ld_y + ch] = y;
                    }
                }
            }
        }
    }
    if (!OUT && live) {
#pragma unroll
        for (int k = 0; k < N; ++k)
            if (k < a.state) states[(ci * a.state + k) * inner + ch] = s[k];
        sums[ci * inner + ch] = sum;
    }
    if (OUT && a.xh && blockIdx.z == gridDim.z - 1)
        for (int t = 0; t < len; ++t) xh_zero_tail(a.xh, a.ncap, row_s[t], (inner + 1) & ~1, tid, SC_THREADS);
}

// pass 2: one thread per (channel, state entry): the state before every chunk, then the slot's new state
__global__ void __launch_bounds__(128) selective_prefix_kernel(DlMambaBatch b, DlSelectiveArgs a, float* __restrict__ states, const float* __restrict__ sums) {
    const int n = blockIdx.x, k = blockIdx.y, ch = blockIdx.z * blockDim.x + threadIdx.x, inner = a.inner, N = a.state;
    if (ch >= inner) return;
    const int s0 = b.seq_start[n], nc = (b.seq_start[n + 1] - s0 + SC - 1) / SC;
    const size_t c0 = s0 / SC + n;
    float* Sg = a.state_pool + ((size_t)b.seq_slot[n] * inner + ch) * N + k;
    const float A = a.A2[(size_t)ch * N + k];
    float R = b.seq_pos0[n] == 0 ? 0.f : *Sg;
    for (int i0 = 0; i0 < nc; i0 += 8) {
        float own[8], sm[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            own[i] = i0 + i < nc ? states[((c0 + i0 + i) * N + k) * inner + ch] : 0.f;
            sm[i] = i0 + i < nc ? sums[(c0 + i0 + i) * inner + ch] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (i0 + i < nc) {
                states[((c0 + i0 + i) * N + k) * inner + ch] = R;
                R = fmaf(ss_ex2(sm[i] * A), R, own[i]);
            }
    }
    *Sg = R;
}

extern "C" int dl_selective_scan_chunked_supported(int state) { return state >= 1 && state <= 32 ? 0 : -1; }

template <int N>
static void launch_selective_chunked(const DlMambaBatch& b, int n_seq, int max_chunks, const DlSelectiveArgs& a, float* states, float* sums, cudaStream_t st) {
    const dim3 grid(n_seq, max_chunks, (a.inner + SC_THREADS - 1) / SC_THREADS);
    selective_chunk_kernel<N, false><<<grid, SC_THREADS, 0, st>>>(b, a, states, sums);
    selective_prefix_kernel<<<dim3(n_seq, a.state, (a.inner + 127) / 128), 128, 0, st>>>(b, a, states, sums);
    selective_chunk_kernel<N, true><<<grid, SC_THREADS, 0, st>>>(b, a, states, sums);
}

extern "C" int dl_selective_scan_chunked(const DlMambaBatch* batch, int n_seq, int max_chunks, const DlSelectiveArgs* args, float* scratch,
                                         int chunk_slots, void* stream) {
    const DlSelectiveArgs& a = *args;
    if (selective_args_ok(a, "dl_selective_scan_chunked")) return -1;
    if (dl_selective_scan_chunked_supported(a.state) != 0 || scratch == nullptr) { dl_set_error("dl_selective_scan_chunked: state %d not supported", a.state); return -1; }
    if (n_seq < 1 || max_chunks < 1) return 0;
    cudaStream_t st = (cudaStream_t)stream;
    float* sums = scratch + (size_t)chunk_slots * a.state * a.inner;
    if (a.state <= 8) launch_selective_chunked<8>(*batch, n_seq, max_chunks, a, scratch, sums, st);
    else if (a.state <= 16) launch_selective_chunked<16>(*batch, n_seq, max_chunks, a, scratch, sums, st);
    else if (a.state <= 24) launch_selective_chunked<24>(*batch, n_seq, max_chunks, a, scratch, sums, st);
    else launch_selective_chunked<32>(*batch, n_seq, max_chunks, a, scratch, sums, st);
    LAYER_CHECK_LAUNCH("dl_selective_scan_chunked");
    return 0;
}
