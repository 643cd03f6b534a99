// Selective scan with a state per channel (Mamba): per channel c and state index n, all f32,
//     step  = softplus(dt_c + dt_bias_c)                       S[c][n] <- exp(-step exp(A_log[c][n])) S[c][n] + step x_c B_n
//     y_c   = sum_n S[c][n] C_n + D_c x_c                      out_c = y_c * silu(z_c)
// A batch is any mix of sequences with one or more consecutive rows each; a sequence whose first row is position 0 starts
// from zeros whatever its slot held.
//
// One kernel for decoding and prompts.  A CTA owns SS_CH channels of one sequence; four neighbouring lanes share a channel and
// keep its state in registers (lane l holds the n with (n / 4) % 4 == l, so that B and C leave shared memory as 16-byte
// words), tokens in order.  The channels are independent and there are thousands of them, so the serial walk over tokens
// still fills the GPU, and every decay e^(step A) is formed exactly once.  SS_TB tokens are staged per barrier pair: step (softplus
// formed once per token and channel), x, B, C; the next tile's global loads are in flight while a tile is walked.  y leaves
// through shared memory, gated, as f32 rows or straight into the next product's bf16 activation image.
#include "layer_common.cuh"
#include "../../../include/dllama_b200.h"

#define SS_CH 32
#define SS_TB 16
#define SS_THREADS (SS_CH * 4)
#define SS_LOG2E 1.4426950408889634f

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
        A[i] = in ? -expf(a.A_log[(size_t)ch * N + k]) * SS_LOG2E : 0.f;      // decays in base 2
    }
    const float Dc = live ? a.D[ch] : 0.f;
    // staging roles: element u of this thread is (token u * 4 + warp, channel lane) and entry (u * SS_THREADS + tid) of B and C
    const int warp = tid >> 5, lane = tid & 31, lch = ch0 + lane;
    const float bias = lch < inner ? a.dt_bias[lch] : 0.f;
    const int r0 = b.seq_start[n], r1 = b.seq_start[n + 1];
    float px[RX], pdt[RX], pB[RB], pC[RB];
    auto fetch = [&](int rb, int buf) {          // row_s[buf] holds the tile's rows (-1: none)
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
    fetch(r0, 0);
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
        if (rb + SS_TB < r1) fetch(rb + SS_TB, buf ^ 1);
#pragma unroll 2
        for (int t = 0; t < nt; ++t) {
            const float dt = dt_s[t][lc], x = x_s[t][lc], dx = dt * x;
            float y0 = 0.f, y1 = 0.f;
#pragma unroll
            for (int i = 0; i < NS; i += 4) {
                const float4 B = *reinterpret_cast<const float4*>(&B_s[t][i * 4 + l * 4]), C = *reinterpret_cast<const float4*>(&C_s[t][i * 4 + l * 4]);
                s[i] = fmaf(exp2f(dt * A[i]), s[i], dx * B.x);              y0 = fmaf(s[i], C.x, y0);
                s[i + 1] = fmaf(exp2f(dt * A[i + 1]), s[i + 1], dx * B.y);  y1 = fmaf(s[i + 1], C.y, y1);
                s[i + 2] = fmaf(exp2f(dt * A[i + 2]), s[i + 2], dx * B.z);  y0 = fmaf(s[i + 2], C.z, y0);
                s[i + 3] = fmaf(exp2f(dt * A[i + 3]), s[i + 3], dx * B.w);  y1 = fmaf(s[i + 3], C.w, y1);
            }
            float y = y0 + y1;
            y += __shfl_xor_sync(0xffffffffu, y, 1);
            y += __shfl_xor_sync(0xffffffffu, y, 2);
            if (l == 0) y_s[t][lc] = fmaf(Dc, x, y);
        }
        __syncthreads();
        // the tile's outputs; (token, group of eight channels) per thread for the image, (token, channel) for rows
        if (a.xh) {
            const int t = tid >> 2, c8 = (tid & 3) * 8;
            if (tid < SS_TB * 4 && t < nt) {
                const int row = row_s[buf][t];
                float v[8];
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const int c = ch0 + c8 + j;
                    v[j] = c < inner ? y_s[t][c8 + j] : 0.f;
                    if (a.z && c < inner) v[j] *= silu_f(a.z[(size_t)row * a.ld_z + c]);
                }
                if (ch0 + c8 < ((inner + 127) & ~127)) {
                    __align__(16) __nv_bfloat16 o[8];
#pragma unroll
                    for (int j = 0; j < 8; ++j) o[j] = __float2bfloat16_rn(v[j]);
                    *reinterpret_cast<uint4*>(a.xh + xh_offset(a.ncap, row, ch0 + c8)) = *reinterpret_cast<const uint4*>(o);
                }
            }
        } else if (lch < inner) {
#pragma unroll
            for (int u = 0; u < RX; ++u) {
                const int t = u * 4 + warp;
                if (t >= nt) break;
                const int row = row_s[buf][t];
                float v = y_s[t][lane];
                if (a.z) v *= silu_f(a.z[(size_t)row * a.ld_z + lch]);
                a.y[(size_t)row * a.ld_y + lch] = v;
            }
        }
        __syncthreads();
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < NS; ++i) {
            const int k = (i >> 2) * 16 + l * 4 + (i & 3);
            if (k < N) Sg[k] = s[i];
        }
    }
    // zeros behind the last channel up to the image's next K tile
    if (a.xh && blockIdx.y == gridDim.y - 1)
        for (int r = r0; r < r1; ++r) {
            const int k0 = (int)gridDim.y * SS_CH + tid;
            if (k0 < ((inner + 127) & ~127)) xh_store(a.xh, a.ncap, b.seq_rows[r], k0, 0.f);
        }
}

extern "C" int dl_selective_scan_supported(int state) { return state >= 1 && state <= 128 ? 0 : -1; }

extern "C" int dl_selective_scan(const DlMambaBatch* batch, int n_seq, const DlSelectiveArgs* args, void* stream) {
    const DlSelectiveArgs& a = *args;
    if (a.inner < 1 || dl_selective_scan_supported(a.state) != 0 || (!a.y && !a.xh)) { dl_set_error("dl_selective_scan: bad shape (inner %d, state %d)", a.inner, a.state); return -1; }
    if (n_seq < 1) return 0;
    cudaStream_t st = (cudaStream_t)stream;
    const dim3 grid(n_seq, (a.inner + SS_CH - 1) / SS_CH);
    if (a.state <= 16) selective_scan_kernel<4><<<grid, SS_THREADS, 0, st>>>(*batch, a);
    else if (a.state <= 32) selective_scan_kernel<8><<<grid, SS_THREADS, 0, st>>>(*batch, a);
    else if (a.state <= 64) selective_scan_kernel<16><<<grid, SS_THREADS, 0, st>>>(*batch, a);
    else selective_scan_kernel<32><<<grid, SS_THREADS, 0, st>>>(*batch, a);
    LAYER_CHECK_LAUNCH("dl_selective_scan");
    return 0;
}
