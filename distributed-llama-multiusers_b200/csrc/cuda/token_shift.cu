// Mixes of every row with the row ahead of it in its sequence:  mix_s[m] = h[m] + (h[m - 1] - h[m]) mu_s,  zeros ahead of the first
// row.  The row ahead of a portion's first row is the slot's carried one.  All mixes leave in one launch, as f32 rows or as the
// bf16 activation images of the products that read them.  The CTA of a sequence's first row of the batch also leaves the
// sequence's last row as the carried one: it is the only reader of what it overwrites.
#include "layer_common.cuh"
#include "../../../include/dllama_b200.h"

#define TS_THREADS 256

__global__ void __launch_bounds__(TS_THREADS) token_shift_kernel(DlMambaBatch b, DlShiftArgs a) {
    const int m = blockIdx.x, W = a.width, tid = threadIdx.x;
    const int n = b.row_seq[m], p = b.pos[m], p0 = b.seq_pos0[n], r0 = b.seq_start[n];
    const bool first = p == p0;
    float* carried = a.state + (size_t)b.seq_slot[n] * W;
    const float* prev = !first ? a.h + (size_t)b.seq_rows[r0 + (p - p0) - 1] * a.ldh : p > 0 ? carried : nullptr;
    const float* last = first ? a.h + (size_t)b.seq_rows[b.seq_start[n + 1] - 1] * a.ldh : nullptr;
    const float* h = a.h + (size_t)m * a.ldh;
    for (int i = tid; i < W; i += TS_THREADS) {
        const float v = h[i], d = (prev ? prev[i] : 0.f) - v;
        if (last) carried[i] = last[i];
        for (int s = 0; s < a.n_mix; ++s) {
            const float x = fmaf(d, a.mu[(size_t)s * W + i], v);
            if (a.xh) xh_store(a.xh + (size_t)s * a.xh_step, a.ncap, m, i, x);
            else a.out[(size_t)s * a.out_step + (size_t)m * a.ld_out + i] = x;
        }
    }
    if (a.xh)
        for (int s = 0; s < a.n_mix; ++s) xh_zero_tail(a.xh + (size_t)s * a.xh_step, a.ncap, m, W, tid, TS_THREADS);
}

// f32 rows with four columns per thread (width % 4 == 0, aligned rows); the CTAs of a row share its columns
__global__ void __launch_bounds__(TS_THREADS) token_shift_vec_kernel(DlMambaBatch b, DlShiftArgs a) {
    const int m = blockIdx.x, W = a.width, i = blockIdx.y * TS_THREADS + threadIdx.x;
    if (i >= W / 4) return;
    const int n = b.row_seq[m], p = b.pos[m], p0 = b.seq_pos0[n], r0 = b.seq_start[n];
    const bool first = p == p0;
    float4* carried = reinterpret_cast<float4*>(a.state + (size_t)b.seq_slot[n] * W);
    const float4* prev = !first ? reinterpret_cast<const float4*>(a.h + (size_t)b.seq_rows[r0 + (p - p0) - 1] * a.ldh) : p > 0 ? carried : nullptr;
    const float4* last = first ? reinterpret_cast<const float4*>(a.h + (size_t)b.seq_rows[b.seq_start[n + 1] - 1] * a.ldh) : nullptr;
    const float4 v = reinterpret_cast<const float4*>(a.h + (size_t)m * a.ldh)[i];
    const float4 q = prev ? prev[i] : make_float4(0.f, 0.f, 0.f, 0.f), d = make_float4(q.x - v.x, q.y - v.y, q.z - v.z, q.w - v.w);
    if (last) carried[i] = last[i];
#pragma unroll 5
    for (int s = 0; s < a.n_mix; ++s) {
        const float4 mu = reinterpret_cast<const float4*>(a.mu + (size_t)s * W)[i];
        reinterpret_cast<float4*>(a.out + (size_t)s * a.out_step + (size_t)m * a.ld_out)[i] =
            make_float4(fmaf(d.x, mu.x, v.x), fmaf(d.y, mu.y, v.y), fmaf(d.z, mu.z, v.z), fmaf(d.w, mu.w, v.w));
    }
}

// images (width % 8 == 0, aligned rows): a warp takes eight rows and four groups of eight columns, so that its 16-byte stores fill 512
// consecutive bytes of an image; groups beyond the width, up to the next 128 columns, are zeros
__global__ void __launch_bounds__(TS_THREADS) token_shift_image_kernel(DlMambaBatch b, DlShiftArgs a, int M) {
    const int m = blockIdx.x * 8 + (threadIdx.x & 7), W = a.width, c = (blockIdx.y * TS_THREADS + threadIdx.x) >> 3;
    if (m >= M || c * 8 >= ((W + 127) & ~127)) return;
    uint8_t* out = a.xh + xh_offset(a.ncap, m, c * 8);
    if (c * 8 >= W) {
        for (int s = 0; s < a.n_mix; ++s) *reinterpret_cast<uint4*>(out + (size_t)s * a.xh_step) = make_uint4(0u, 0u, 0u, 0u);
        return;
    }
    const int n = b.row_seq[m], p = b.pos[m], p0 = b.seq_pos0[n], r0 = b.seq_start[n];
    const bool first = p == p0;
    float4* carried = reinterpret_cast<float4*>(a.state + (size_t)b.seq_slot[n] * W);
    const float4* prev = !first ? reinterpret_cast<const float4*>(a.h + (size_t)b.seq_rows[r0 + (p - p0) - 1] * a.ldh) : p > 0 ? carried : nullptr;
    const float4* last = first ? reinterpret_cast<const float4*>(a.h + (size_t)b.seq_rows[b.seq_start[n + 1] - 1] * a.ldh) : nullptr;
    float4 v[2], d[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        const int i = c * 2 + x;
        v[x] = reinterpret_cast<const float4*>(a.h + (size_t)m * a.ldh)[i];
        const float4 q = prev ? prev[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        d[x] = make_float4(q.x - v[x].x, q.y - v[x].y, q.z - v[x].z, q.w - v[x].w);
        if (last) carried[i] = last[i];
    }
#pragma unroll 5
    for (int s = 0; s < a.n_mix; ++s) {
        uint32_t w[4];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const float4 mu = reinterpret_cast<const float4*>(a.mu + (size_t)s * W)[c * 2 + x];
            __nv_bfloat162 lo = __floats2bfloat162_rn(fmaf(d[x].x, mu.x, v[x].x), fmaf(d[x].y, mu.y, v[x].y));
            __nv_bfloat162 hi = __floats2bfloat162_rn(fmaf(d[x].z, mu.z, v[x].z), fmaf(d[x].w, mu.w, v[x].w));
            w[2 * x] = *reinterpret_cast<uint32_t*>(&lo);
            w[2 * x + 1] = *reinterpret_cast<uint32_t*>(&hi);
        }
        *reinterpret_cast<uint4*>(out + (size_t)s * a.xh_step) = make_uint4(w[0], w[1], w[2], w[3]);
    }
}

extern "C" int dl_token_shift(const DlMambaBatch* batch, int M, const DlShiftArgs* args, void* stream) {
    const DlShiftArgs& a = *args;
    if (M < 1 || a.width < 1 || a.n_mix < 1 || !a.h || !a.mu || !a.state || (!a.out && !a.xh)) { dl_set_error("dl_token_shift: bad arguments"); return -1; }
    const auto al = [](const void* p, long long ld) { return ((uintptr_t)p & 15) == 0 && ld % 4 == 0; };
    const bool vec = a.width % 4 == 0 && al(a.h, a.ldh) && al(a.mu, 0) && al(a.state, 0) && al(a.out, a.ld_out) && a.out_step % 4 == 0 && al(a.xh, 0) && a.xh_step % 16 == 0;
    if (vec && !a.xh) token_shift_vec_kernel<<<dim3(M, (a.width / 4 + TS_THREADS - 1) / TS_THREADS), TS_THREADS, 0, (cudaStream_t)stream>>>(*batch, a);
    else if (vec && a.width % 8 == 0) token_shift_image_kernel<<<dim3((M + 7) / 8, ((a.width + 127) / 128 * 16 + 31) / 32), TS_THREADS, 0, (cudaStream_t)stream>>>(*batch, a, M);
    else token_shift_kernel<<<M, TS_THREADS, 0, (cudaStream_t)stream>>>(*batch, a);
    LAYER_CHECK_LAUNCH("dl_token_shift");
    return 0;
}
