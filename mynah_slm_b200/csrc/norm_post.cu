// RMS norms that stand BEHIND a sublayer:
//
//   rmsnorm_add      x <- x (+ e) + y / sqrt(mean(y^2) + eps) * gain          (x fp32 in place, y fp32)
//                    and, when asked, the norm of the new x in the same pass:
//                    h = x / sqrt(mean(x^2) + eps2) * gain2                     (h fp32)
//                    e, optional, is another fp32 row added on the way (an input fed back in).
//                    A bfloat16 copy of the new x can be left too (the next sublayer's input where it reads x itself).
//   rms_rows         out = x / sqrt(mean(x^2) + eps) * gain                    (x, out in the activation type; x a column slice)
//   rms_pair_mean    out = weight * (a / rms(a) * ga + b / rms(b) * gb)        (a, b, out fp32)
//
// All sums are fp32 and run in an order fixed by the thread layout. A CTA takes one row; the row stays in
// registers between its two passes while it has at most 8 values a thread.
#include "common.cuh"

namespace {

constexpr int NP_THREADS = 256;
constexpr int NP_KEEP = 8;

__global__ void __launch_bounds__(NP_THREADS)
rmsnorm_add_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ extra, VecRef gain,
                   float eps, VecRef gain2, float eps2, float* __restrict__ h, bf16* __restrict__ copy, int D) {
    __shared__ float red[32];
    griddep_launch_small();
    griddep_wait();
    const size_t row = (size_t)blockIdx.x * D;
    const bool keep = D <= NP_KEEP * NP_THREADS;
    float v[NP_KEEP];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NP_KEEP; i++) {
        const int d = threadIdx.x + i * NP_THREADS;
        v[i] = d < D ? y[row + d] : 0.f;
        ss = fmaf(v[i], v[i], ss);
    }
    if (!keep)
        for (int d = threadIdx.x + NP_KEEP * NP_THREADS; d < D; d += NP_THREADS) ss = fmaf(y[row + d], y[row + d], ss);
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)D + eps);
    float s2 = 0.f;
#pragma unroll
    for (int i = 0; i < NP_KEEP; i++) {
        const int d = threadIdx.x + i * NP_THREADS;
        if (d < D) {
            float nx = x[row + d];
            if (extra != nullptr) nx += extra[row + d];
            nx += v[i] * r * gain.at(d);
            x[row + d] = nx;
            if (copy != nullptr) copy[row + d] = __float2bfloat16_rn(nx);
            v[i] = nx;
            s2 = fmaf(nx, nx, s2);
        }
    }
    if (!keep)
        for (int d = threadIdx.x + NP_KEEP * NP_THREADS; d < D; d += NP_THREADS) {
            float nx = x[row + d];
            if (extra != nullptr) nx += extra[row + d];
            nx += y[row + d] * r * gain.at(d);
            x[row + d] = nx;
            if (copy != nullptr) copy[row + d] = __float2bfloat16_rn(nx);
            s2 = fmaf(nx, nx, s2);
        }
    if (h == nullptr) return;
    const float r2 = 1.0f / sqrtf(block_sum(s2, red) / (float)D + eps2);
#pragma unroll
    for (int i = 0; i < NP_KEEP; i++) {
        const int d = threadIdx.x + i * NP_THREADS;
        if (d < D) h[row + d] = v[i] * r2 * gain2.at(d);
    }
    if (!keep)
        for (int d = threadIdx.x + NP_KEEP * NP_THREADS; d < D; d += NP_THREADS) h[row + d] = x[row + d] * r2 * gain2.at(d);
}

// The same for rows of a multiple of 4 values, up to 4 * 1024 (and no second norm): four values a thread, in 16-byte accesses.
__global__ void __launch_bounds__(1024)
rmsnorm_add_vec4_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ extra, VecRef gain, float eps,
                        bf16* __restrict__ copy, int D) {
    __shared__ float red[32];
    griddep_launch_small();
    griddep_wait();
    const int d = threadIdx.x * 4;
    const bool on = d < D;
    const size_t at = (size_t)blockIdx.x * D + d;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f), w = v;
    if (on) {
        v = *reinterpret_cast<const float4*>(y + at);
        w = *reinterpret_cast<const float4*>(x + at);
        if (extra != nullptr) {
            const float4 e = *reinterpret_cast<const float4*>(extra + at);
            w.x += e.x; w.y += e.y; w.z += e.z; w.w += e.w;
        }
    }
    const float ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)D + eps);
    if (!on) return;
    w.x += v.x * r * gain.at(d);
    w.y += v.y * r * gain.at(d + 1);
    w.z += v.z * r * gain.at(d + 2);
    w.w += v.w * r * gain.at(d + 3);
    *reinterpret_cast<float4*>(x + at) = w;
    if (copy != nullptr) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(w.x, w.y), b = __floats2bfloat162_rn(w.z, w.w);
        *reinterpret_cast<uint2*>(copy + at) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    }
}

// one CTA a row of n values, rows ld_x and ld_o apart
template <typename T>
__global__ void __launch_bounds__(128)
rms_rows_kernel(const T* __restrict__ x, int ld_x, VecRef gain, float eps, T* __restrict__ out, int ld_o, int n) {
    __shared__ float red[32];
    griddep_launch_small();
    griddep_wait();
    const T* row = x + (size_t)blockIdx.x * ld_x;
    constexpr int KEEP = 8;
    float v[KEEP];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; i++) {
        const int d = threadIdx.x + i * 128;
        v[i] = d < n ? to_f32(row[d]) : 0.f;
        ss = fmaf(v[i], v[i], ss);
    }
    for (int d = threadIdx.x + KEEP * 128; d < n; d += 128) {
        const float u = to_f32(row[d]);
        ss = fmaf(u, u, ss);
    }
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)n + eps);
    T* o = out + (size_t)blockIdx.x * ld_o;
#pragma unroll
    for (int i = 0; i < KEEP; i++) {
        const int d = threadIdx.x + i * 128;
        if (d < n) o[d] = from_f32<T>(v[i] * r * gain.at(d));
    }
    for (int d = threadIdx.x + KEEP * 128; d < n; d += 128) o[d] = from_f32<T>(to_f32(row[d]) * r * gain.at(d));
}

__global__ void __launch_bounds__(NP_THREADS)
rms_pair_mean_kernel(const float* __restrict__ a, const float* __restrict__ b, VecRef ga, VecRef gb, float eps,
                     float weight, float* __restrict__ out, int D) {
    __shared__ float red[32];
    griddep_launch_small();
    griddep_wait();
    const size_t row = (size_t)blockIdx.x * D;
    float sa = 0.f, sb = 0.f;
    for (int d = threadIdx.x; d < D; d += NP_THREADS) {
        sa = fmaf(a[row + d], a[row + d], sa);
        sb = fmaf(b[row + d], b[row + d], sb);
    }
    const float ra = 1.0f / sqrtf(block_sum(sa, red) / (float)D + eps);
    const float rb = 1.0f / sqrtf(block_sum(sb, red) / (float)D + eps);
    for (int d = threadIdx.x; d < D; d += NP_THREADS)
        out[row + d] = weight * (a[row + d] * ra * ga.at(d) + b[row + d] * rb * gb.at(d));
}

}  // namespace

// x [T, D] fp32 in place; y [T, D] fp32; extra null or [T, D] fp32; gain [D] in g_dtype. h null, or [T, D] fp32 that
// receives the norm of the new x with gain2 [D] (g2_dtype) and eps2. copy null, or bf16 [T, D] that receives the new x.
MYNAH_API int mynah_rmsnorm_add(float* x, const float* y, const float* extra, const void* gain, int g_dtype, float eps,
                                const void* gain2, int g2_dtype, float eps2, float* h, void* copy, int T, int D, cudaStream_t stream) {
    if (T == 0) return 0;
    MYNAH_REQUIRE(T > 0 && D > 0, "rmsnorm_add: bad sizes T=%d D=%d", T, D);
    MYNAH_REQUIRE(h == nullptr || gain2 != nullptr, "rmsnorm_add: a second norm needs its gain");
    if (h == nullptr && D % 4 == 0 && D <= 4096 && (((uintptr_t)x | (uintptr_t)y | (uintptr_t)extra) & 15) == 0 && ((uintptr_t)copy & 7) == 0) {
        mynah_launch(rmsnorm_add_vec4_kernel, dim3(T), dim3((D / 4 + 31) / 32 * 32), 0, stream, x, y, extra, VecRef{gain, g_dtype}, eps,
                     (bf16*)copy, D);
        return mynah_check_launch("rmsnorm_add");
    }
    mynah_launch(rmsnorm_add_kernel, dim3(T), dim3(NP_THREADS), 0, stream, x, y, extra, VecRef{gain, g_dtype}, eps,
                 VecRef{gain2, g2_dtype}, eps2, h, (bf16*)copy, D);
    return mynah_check_launch("rmsnorm_add");
}

// x: [T] rows of n values, ld_x apart (a column slice of wider rows), in dtype; gain [n] in g_dtype; out [T] rows, ld_o apart.
MYNAH_API int mynah_rms_rows(const void* x, int dtype, int ld_x, const void* gain, int g_dtype, float eps, void* out, int ld_o, int T,
                             int n, cudaStream_t stream) {
    if (T == 0) return 0;
    MYNAH_REQUIRE(T > 0 && n > 0 && ld_x >= n && ld_o >= n, "rms_rows: bad sizes T=%d n=%d", T, n);
    if (dtype == MYNAH_F32)
        mynah_launch(rms_rows_kernel<float>, dim3(T), dim3(128), 0, stream, (const float*)x, ld_x, VecRef{gain, g_dtype}, eps, (float*)out, ld_o, n);
    else if (dtype == MYNAH_BF16)
        mynah_launch(rms_rows_kernel<bf16>, dim3(T), dim3(128), 0, stream, (const bf16*)x, ld_x, VecRef{gain, g_dtype}, eps, (bf16*)out, ld_o, n);
    else
        return mynah_fail("rms_rows: unsupported dtype %d", dtype);
    return mynah_check_launch("rms_rows");
}

// a, b, out [T, D] fp32; ga, gb [D] in g_dtype.
MYNAH_API int mynah_rms_pair_mean(const float* a, const float* b, const void* ga, const void* gb, int g_dtype, float eps,
                                  float weight, float* out, int T, int D, cudaStream_t stream) {
    if (T == 0) return 0;
    MYNAH_REQUIRE(T > 0 && D > 0, "rms_pair_mean: bad sizes T=%d D=%d", T, D);
    mynah_launch(rms_pair_mean_kernel, dim3(T), dim3(NP_THREADS), 0, stream, a, b, VecRef{ga, g_dtype}, VecRef{gb, g_dtype},
                 eps, weight, out, D);
    return mynah_check_launch("rms_pair_mean");
}
