// RMS normalisation in its variants, all in f32:  y = v / sqrt(mean(v^2) + eps) * scale
//   * scale = w  or  (1 + w)  (a weight stored around zero)  or 1 (no weight);
//   * the row may be normalised in `groups` equal parts, each by its own root mean square;
//   * v = x  or  x * silu(gate)  (a gate applied before the norm);
//   * the result is stored, or added to what y holds (a norm on a sublayer's output, summed into the residual stream);
//   * an optional row map gathers source rows (the final norm of the rows whose logits are wanted).
// One CTA per (row, group); groups of up to 4096 values stay in registers between the sum of squares and the scaling.
#include "layer_common.cuh"
#include "../../../include/dllama_b200.h"

#define RN_THREADS 256
#define RN_CACHE 16                // values a thread keeps in registers between the two passes (groups of up to 4096)

__global__ void __launch_bounds__(RN_THREADS) rms_norm_kernel(DlNormArgs a) {
    __shared__ float red[32];
    const int m = blockIdx.x, g = blockIdx.y;
    const int src = a.rows ? a.rows[m] : m;
    const int gd = a.dim / a.groups;
    const float* x = a.x + (size_t)src * a.ldx + (size_t)g * gd;
    const float* gate = a.gate ? a.gate + (size_t)src * a.ld_gate + (size_t)g * gd : nullptr;
    const bool cached = gd <= RN_THREADS * RN_CACHE;
    float v[RN_CACHE];
    float ss = 0.f;
    if (cached) {
#pragma unroll
        for (int k = 0; k < RN_CACHE; ++k) {
            const int i = threadIdx.x + k * RN_THREADS;
            float t = 0.f;
            if (i < gd) {
                t = x[i];
                if (gate) t *= silu_f(gate[i]);
            }
            v[k] = t;
            ss = fmaf(t, t, ss);
        }
    } else {
        for (int i = threadIdx.x; i < gd; i += RN_THREADS) {
            float t = x[i];
            if (gate) t *= silu_f(gate[i]);
            ss = fmaf(t, t, ss);
        }
    }
    ss = block_sum(ss, red);
    const float inv = 1.f / sqrtf(ss / (float)gd + a.eps);
    float* y = a.y + (size_t)m * a.ldy + (size_t)g * gd;
    const float* w = a.w ? a.w + (size_t)g * gd : nullptr;
    if (cached) {
#pragma unroll
        for (int k = 0; k < RN_CACHE; ++k) {
            const int i = threadIdx.x + k * RN_THREADS;
            if (i < gd) {
                float t = v[k] * inv;
                if (w) t *= a.plus_one ? 1.f + w[i] : w[i];
                y[i] = a.accumulate ? y[i] + t : t;
            }
        }
    } else {
        for (int i = threadIdx.x; i < gd; i += RN_THREADS) {
            float t = x[i];
            if (gate) t *= silu_f(gate[i]);
            t *= inv;
            if (w) t *= a.plus_one ? 1.f + w[i] : w[i];
            y[i] = a.accumulate ? y[i] + t : t;
        }
    }
}

extern "C" int dl_rms_norm(const DlNormArgs* args, void* stream) {
    const DlNormArgs& a = *args;
    if (a.M < 1 || a.dim < 1 || a.groups < 1 || a.dim % a.groups != 0) { dl_set_error("dl_rms_norm: bad shape"); return -1; }
    if (a.accumulate && (const float*)a.y == a.x) { dl_set_error("dl_rms_norm: accumulate needs y != x"); return -1; }
    dim3 grid(a.M, a.groups);
    rms_norm_kernel<<<grid, RN_THREADS, 0, (cudaStream_t)stream>>>(a);
    LAYER_CHECK_LAUNCH("dl_rms_norm");
    return 0;
}

// ------------------------------------------------------------------------------------------------
// PolyNorm: y = c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3, N(u) = u / sqrt(mean(u^2) + eps), powers element by element.
// One CTA per row: the sums of z^2, z^4 and z^6 in one pass (the row stays in registers up to 4096 values), then the
// three scalings.
// ------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(RN_THREADS) poly_norm_kernel(const float* __restrict__ x, long long ldx, float* __restrict__ y, long long ldy,
                                                               int dim, const float* __restrict__ coef, float eps) {
    __shared__ float red[32];
    const int m = blockIdx.x;
    const float* xr = x + (size_t)m * ldx;
    const bool cached = dim <= RN_THREADS * RN_CACHE;
    float v[RN_CACHE];
    float s2 = 0.f, s4 = 0.f, s6 = 0.f;
    if (cached) {
#pragma unroll
        for (int k = 0; k < RN_CACHE; ++k) {
            const int i = threadIdx.x + k * RN_THREADS;
            const float t = i < dim ? xr[i] : 0.f;
            v[k] = t;
            const float t2 = t * t, t3 = t2 * t;
            s2 = fmaf(t, t, s2); s4 = fmaf(t2, t2, s4); s6 = fmaf(t3, t3, s6);
        }
    } else {
        for (int i = threadIdx.x; i < dim; i += RN_THREADS) {
            const float t = xr[i], t2 = t * t, t3 = t2 * t;
            s2 = fmaf(t, t, s2); s4 = fmaf(t2, t2, s4); s6 = fmaf(t3, t3, s6);
        }
    }
    s2 = block_sum(s2, red);
    s4 = block_sum(s4, red);
    s6 = block_sum(s6, red);
    const float c1 = coef[0] / sqrtf(s2 / (float)dim + eps), c2 = coef[1] / sqrtf(s4 / (float)dim + eps),
                c3 = coef[2] / sqrtf(s6 / (float)dim + eps), c0 = coef[3];
    float* yr = y + (size_t)m * ldy;
    if (cached) {
#pragma unroll
        for (int k = 0; k < RN_CACHE; ++k) {
            const int i = threadIdx.x + k * RN_THREADS;
            if (i < dim) { const float t = v[k]; yr[i] = fmaf(t, fmaf(t, fmaf(t, c3, c2), c1), c0); }
        }
    } else {
        for (int i = threadIdx.x; i < dim; i += RN_THREADS) { const float t = xr[i]; yr[i] = fmaf(t, fmaf(t, fmaf(t, c3, c2), c1), c0); }
    }
}

extern "C" int dl_poly_norm(const float* x, long long ldx, float* y, long long ldy, int M, int dim, const float* coef, float eps,
                            void* stream) {
    if (M < 1 || dim < 1 || coef == nullptr) { dl_set_error("dl_poly_norm: bad shape"); return -1; }
    poly_norm_kernel<<<M, RN_THREADS, 0, (cudaStream_t)stream>>>(x, ldx, y, ldy, dim, coef, eps);
    LAYER_CHECK_LAUNCH("dl_poly_norm");
    return 0;
}

// ------------------------------------------------------------------------------------------------
// One step of a residual stream: a row's sum (the stream, plain or scaled terms, terms normalised first, a vector for every row),
// then up to two normed copies of it (root mean square, or layer norm with bias), as f32 rows or straight into the bf16 activation image of the products that read them.  One
// CTA per row; the row stays in shared memory between the sums.  Three dependent passes at most: the roots of the normalised
// terms, the sum and its root, the copies.
// ------------------------------------------------------------------------------------------------
#define RS_THREADS 256
__global__ void __launch_bounds__(RS_THREADS) residual_step_kernel(DlResidualArgs a) {
    extern __shared__ __align__(16) float row_s[];           // [dim], then a and b's rows when they are there
    __shared__ float red[32];
    const int m = blockIdx.x, dim = a.dim, tid = threadIdx.x;
    const size_t src = a.rows ? a.rows[m] : m;
    const float* xi = a.x_in ? a.x_in + src * a.ld_in : nullptr;
    float inv_a = 0.f, inv_b = 0.f;
    float* ra = row_s + dim;
    float* rb = ra + dim;
    if (a.norm_a) {
        const float* pa = a.norm_a + src * a.ld_a;
        const float* pb = a.norm_b ? a.norm_b + src * a.ld_b : nullptr;
        float sa = 0.f, sb = 0.f;
#pragma unroll 4
        for (int i = tid; i < dim; i += RS_THREADS) {
            const float u = pa[i], v = pb ? pb[i] : 0.f;
            ra[i] = u;
            if (pb) rb[i] = v;
            sa = fmaf(u, u, sa);
            sb = fmaf(v, v, sb);
        }
        inv_a = 1.f / sqrtf(block_sum(sa, red) / (float)dim + a.eps);
        if (pb) inv_b = 1.f / sqrtf(block_sum(sb, red) / (float)dim + a.eps);
    }
    const __nv_bfloat16* tb = a.table ? (const __nv_bfloat16*)a.table + src * a.ld_in : nullptr;
    const float* p1 = a.add1 ? a.add1 + src * a.ld_add1 : nullptr;
    const float* p2 = a.add2 ? a.add2 + src * a.ld_add2 : nullptr;
    const float* p3 = a.add3 ? a.add3 + src * a.ld_add3 : nullptr;
    float ss = 0.f;
#pragma unroll 4
    for (int i = tid; i < dim; i += RS_THREADS) {            // a thread meets only its own columns again: no barrier for row_s, ra, rb
        float t = 0.f;
        if (a.norm_a) {
            t = a.w_a[i] * (ra[i] * inv_a);
            if (a.norm_b) t = fmaf(a.w_b[i], rb[i] * inv_b, t);
        }
        if (p1) t += a.add_scaled ? a.scale1 * p1[i] : p1[i];
        if (p2) t += a.add_scaled ? a.scale2 * p2[i] : p2[i];
        if (p3) t += p3[i];
        if (xi) t += xi[i];
        if (tb) t += __bfloat162float(tb[i]);
        if (a.vec) t += a.vec[i];
        row_s[i] = t;
        if (a.x) a.x[(size_t)m * a.ldx + i] = t;
        ss = a.layer_norm ? ss + t : fmaf(t, t, ss);
    }
    if (!a.w1) return;
    ss = block_sum(ss, red) / (float)dim;
    float mean = 0.f;
    if (a.layer_norm) {
        mean = ss;
        float sc = 0.f;
        for (int i = tid; i < dim; i += RS_THREADS) { const float c = row_s[i] - mean; sc = fmaf(c, c, sc); }
        ss = block_sum(sc, red) / (float)dim;
    }
    const float inv = 1.f / sqrtf(ss + a.eps);
#pragma unroll 4
    for (int i = tid; i < dim; i += RS_THREADS) {
        const float t = (row_s[i] - mean) * inv;
        const float u = fmaf(t, a.w1[i], a.b1 ? a.b1[i] : 0.f);
        if (a.xh1) xh_store(a.xh1, a.ncap, m, i, u); else a.h1[(size_t)m * a.ldh + i] = u;
        if (a.w2) {
            const float v = fmaf(t, a.w2[i], a.b2 ? a.b2[i] : 0.f);
            if (a.xh2) xh_store(a.xh2, a.ncap, m, i, v); else a.h2[(size_t)m * a.ldh + i] = v;
        }
    }
    if (a.xh1) xh_zero_tail(a.xh1, a.ncap, m, dim, tid, RS_THREADS);
    if (a.xh2) xh_zero_tail(a.xh2, a.ncap, m, dim, tid, RS_THREADS);
}

// the same with four columns per thread and step (dim % 4 == 0, aligned rows): every term of the row is loaded at once and stays in
// registers, so a decoded row costs one round of loads and two block sums
__device__ __forceinline__ float4 rs_add(float4 x, float4 y) { return make_float4(x.x + y.x, x.y + y.y, x.z + y.z, x.w + y.w); }
__device__ __forceinline__ float rs_sq(float4 x, float acc) { return fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, fmaf(x.w, x.w, acc)))); }
__device__ __forceinline__ void rs_put(float* h, uint8_t* xh, int ncap, int m, long long ld, int i, float4 v) {
    if (xh) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
        *reinterpret_cast<uint2*>(xh + xh_offset(ncap, m, i * 4)) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
    } else {
        reinterpret_cast<float4*>(h + (size_t)m * ld)[i] = v;
    }
}

template <int NG>
__global__ void __launch_bounds__(RS_THREADS) residual_step_vec_kernel(DlResidualArgs a) {
    __shared__ float red[2 * (RS_THREADS / 32)];
    const int m = blockIdx.x, dim = a.dim, n4 = dim >> 2, tid = threadIdx.x;
    const size_t src = a.rows ? a.rows[m] : m;
    float4 t[NG], u[NG], v[NG];
    float sa = 0.f, sb = 0.f;
#pragma unroll
    for (int k = 0; k < NG; ++k) {
        const int i = tid + k * RS_THREADS;
        t[k] = u[k] = v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < n4) {
            if (a.norm_a) u[k] = reinterpret_cast<const float4*>(a.norm_a + src * a.ld_a)[i];
            if (a.norm_b) v[k] = reinterpret_cast<const float4*>(a.norm_b + src * a.ld_b)[i];
            if (a.add1) t[k] = reinterpret_cast<const float4*>(a.add1 + src * a.ld_add1)[i];
            if (a.add_scaled) t[k] = make_float4(a.scale1 * t[k].x, a.scale1 * t[k].y, a.scale1 * t[k].z, a.scale1 * t[k].w);
            if (a.add2) {
                const float4 w = reinterpret_cast<const float4*>(a.add2 + src * a.ld_add2)[i];
                const float s = a.add_scaled ? a.scale2 : 1.f;
                t[k] = make_float4(fmaf(s, w.x, t[k].x), fmaf(s, w.y, t[k].y), fmaf(s, w.z, t[k].z), fmaf(s, w.w, t[k].w));
            }
            if (a.x_in) t[k] = rs_add(t[k], reinterpret_cast<const float4*>(a.x_in + src * a.ld_in)[i]);
            if (a.table) {
                const uint2 w = reinterpret_cast<const uint2*>((const __nv_bfloat16*)a.table + src * a.ld_in)[i];
                t[k] = rs_add(t[k], make_float4(__uint_as_float(w.x << 16), __uint_as_float(w.x & 0xffff0000u), __uint_as_float(w.y << 16), __uint_as_float(w.y & 0xffff0000u)));
            }
            if (a.add3) t[k] = rs_add(t[k], reinterpret_cast<const float4*>(a.add3 + src * a.ld_add3)[i]);
            if (a.vec) t[k] = rs_add(t[k], reinterpret_cast<const float4*>(a.vec)[i]);
        }
        sa = rs_sq(u[k], sa);
        sb = rs_sq(v[k], sb);
    }
    const int warp = tid >> 5, lane = tid & 31;
    if (a.norm_a) {
        sa = warp_sum(sa);
        sb = warp_sum(sb);
        if (lane == 0) { red[warp] = sa; red[RS_THREADS / 32 + warp] = sb; }
        __syncthreads();
        sa = sb = 0.f;
#pragma unroll
        for (int w = 0; w < RS_THREADS / 32; ++w) { sa += red[w]; sb += red[RS_THREADS / 32 + w]; }
        const float ia = 1.f / sqrtf(sa / (float)dim + a.eps), ib = 1.f / sqrtf(sb / (float)dim + a.eps);
#pragma unroll
        for (int k = 0; k < NG; ++k) {
            const int i = tid + k * RS_THREADS;
            if (i < n4) {
                const float4 wa = reinterpret_cast<const float4*>(a.w_a)[i];
                float4 n = make_float4(wa.x * (u[k].x * ia), wa.y * (u[k].y * ia), wa.z * (u[k].z * ia), wa.w * (u[k].w * ia));
                if (a.norm_b) {
                    const float4 wb = reinterpret_cast<const float4*>(a.w_b)[i];
                    n = make_float4(fmaf(wb.x, v[k].x * ib, n.x), fmaf(wb.y, v[k].y * ib, n.y), fmaf(wb.z, v[k].z * ib, n.z), fmaf(wb.w, v[k].w * ib, n.w));
                }
                t[k] = rs_add(n, t[k]);
            }
        }
        __syncthreads();
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NG; ++k) {
        const int i = tid + k * RS_THREADS;
        if (a.x && i < n4) reinterpret_cast<float4*>(a.x + (size_t)m * a.ldx)[i] = t[k];
        ss = a.layer_norm ? ss + (t[k].x + t[k].y) + (t[k].z + t[k].w) : rs_sq(t[k], ss);
    }
    if (!a.w1) return;
    if (a.layer_norm) {                       // the row minus its mean, then the sum of ITS squares
        ss = warp_sum(ss);
        if (lane == 0) red[RS_THREADS / 32 + warp] = ss;
        __syncthreads();
        float mean = 0.f;
#pragma unroll
        for (int w = 0; w < RS_THREADS / 32; ++w) mean += red[RS_THREADS / 32 + w];
        mean /= (float)dim;
        ss = 0.f;
#pragma unroll
        for (int k = 0; k < NG; ++k)
            if (tid + k * RS_THREADS < n4) {
                t[k] = make_float4(t[k].x - mean, t[k].y - mean, t[k].z - mean, t[k].w - mean);
                ss = rs_sq(t[k], ss);
            }
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < RS_THREADS / 32; ++w) ss += red[w];
    const float inv = 1.f / sqrtf(ss / (float)dim + a.eps);
#pragma unroll
    for (int k = 0; k < NG; ++k) {
        const int i = tid + k * RS_THREADS;
        if (i < n4) {
            const float4 w = reinterpret_cast<const float4*>(a.w1)[i];
            const float4 n = make_float4(t[k].x * inv, t[k].y * inv, t[k].z * inv, t[k].w * inv);
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f), b1 = a.b1 ? reinterpret_cast<const float4*>(a.b1)[i] : zero;
            rs_put(a.h1, a.xh1, a.ncap, m, a.ldh, i, make_float4(fmaf(n.x, w.x, b1.x), fmaf(n.y, w.y, b1.y), fmaf(n.z, w.z, b1.z), fmaf(n.w, w.w, b1.w)));
            if (a.w2) {
                const float4 w2 = reinterpret_cast<const float4*>(a.w2)[i];
                const float4 b2 = a.b2 ? reinterpret_cast<const float4*>(a.b2)[i] : zero;
                rs_put(a.h2, a.xh2, a.ncap, m, a.ldh, i, make_float4(fmaf(n.x, w2.x, b2.x), fmaf(n.y, w2.y, b2.y), fmaf(n.z, w2.z, b2.z), fmaf(n.w, w2.w, b2.w)));
            }
        }
    }
    if (a.xh1) xh_zero_tail(a.xh1, a.ncap, m, dim, tid, RS_THREADS);
    if (a.xh2) xh_zero_tail(a.xh2, a.ncap, m, dim, tid, RS_THREADS);
}

extern "C" int dl_residual_step(const DlResidualArgs* args, void* stream) {
    const DlResidualArgs& a = *args;
    if (a.M < 1 || a.dim < 1) { dl_set_error("dl_residual_step: bad shape"); return -1; }
    if ((a.norm_b && !a.norm_a) || (a.norm_a && !a.w_a) || (a.norm_b && !a.w_b) || (a.w2 && !a.w1) || (a.w1 && !a.h1 && !a.xh1) || (a.w2 && !a.h2 && !a.xh2)) {
        dl_set_error("dl_residual_step: terms do not fit together");
        return -1;
    }
    if (a.x_in && a.table) { dl_set_error("dl_residual_step: x_in and table"); return -1; }
    const auto al = [](const void* p, long long ld) { return ((uintptr_t)p & 15) == 0 && ld % 4 == 0; };
    const bool vec = a.dim % 4 == 0 && a.dim <= 4 * RS_THREADS * 8 && al(a.x_in, a.ld_in) && al(a.table, a.ld_in) && al(a.add1, a.ld_add1) && al(a.add2, a.ld_add2) &&
                     al(a.add3, a.ld_add3) && al(a.norm_a, a.ld_a) && al(a.norm_b, a.ld_b) && al(a.w_a, 0) && al(a.w_b, 0) && al(a.vec, 0) && al(a.x, a.ldx) &&
                     al(a.w1, 0) && al(a.w2, 0) && al(a.b1, 0) && al(a.b2, 0) && al(a.h1, a.ldh) && al(a.h2, a.ldh);
    if (vec) {
        cudaStream_t st = (cudaStream_t)stream;
        if (a.dim <= 4 * RS_THREADS) residual_step_vec_kernel<1><<<a.M, RS_THREADS, 0, st>>>(a);
        else if (a.dim <= 8 * RS_THREADS) residual_step_vec_kernel<2><<<a.M, RS_THREADS, 0, st>>>(a);
        else if (a.dim <= 16 * RS_THREADS) residual_step_vec_kernel<4><<<a.M, RS_THREADS, 0, st>>>(a);
        else residual_step_vec_kernel<8><<<a.M, RS_THREADS, 0, st>>>(a);
        LAYER_CHECK_LAUNCH("dl_residual_step");
        return 0;
    }
    const size_t smem = (size_t)a.dim * (1 + (a.norm_a ? 1 : 0) + (a.norm_b ? 1 : 0)) * sizeof(float);
    if (smem > 200 * 1024) { dl_set_error("dl_residual_step: rows of %d do not fit shared memory", a.dim); return -1; }
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(residual_step_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) { dl_set_error("dl_residual_step: shared memory attribute: %s", cudaGetErrorString(e)); return -(int)e; }
    }
    residual_step_kernel<<<a.M, RS_THREADS, smem, (cudaStream_t)stream>>>(a);
    LAYER_CHECK_LAUNCH("dl_residual_step");
    return 0;
}
