// Row-wise kernels around the matrix products: token embedding, RMSNorm with
// the residual add folded in, SwiGLU, and the plain residual add.
//
// The residual stream is fp32 in both precisions. Sums of squares and the
// scale are fp32; the order of every sum is fixed by the thread layout, so a
// row's result does not depend on which other rows share the launch.
#include "common.cuh"
#include "layout.cuh"
#include "head_prep.cuh"

// ------------------------------------------------------------- embedding
// x[t, :] = E[token_t, :] * scale   (mynah-slm src/arch_qwen3.c:186 has no scaling: scale 1; a design that
// multiplies its embedding by a constant gives it here; the product is fp32)
template <typename TW>
__global__ void embed_gather_kernel(const TW* __restrict__ table, const int* __restrict__ tokens,
                                    float* __restrict__ x, int D, int V, float scale) {
    griddep_launch();
    griddep_wait();
    const int t = blockIdx.x;
    const int tok = tokens[t];
    float* out = x + (size_t)t * D;
    if (tok < 0 || tok >= V) {      // refused on the host already; never read out of range
        for (int i = threadIdx.x; i < D; i += blockDim.x) out[i] = 0.f;
        return;
    }
    const TW* row = table + (size_t)tok * D;
    for (int i = threadIdx.x; i < D; i += blockDim.x) out[i] = to_f32(row[i]) * scale;
}

MYNAH_API int mynah_embed_gather(const void* table, int table_dtype, const int* tokens, float* x,
                                 int T, int D, int V, float scale, cudaStream_t stream) {
    if (T == 0) return 0;
    MYNAH_REQUIRE(T > 0 && D > 0 && V > 0, "embed_gather: bad sizes T=%d D=%d V=%d", T, D, V);
    const int threads = D >= 1024 ? 256 : (D >= 256 ? 128 : 64);
    if (table_dtype == MYNAH_F32)
        mynah_launch(embed_gather_kernel<float>, dim3(T), dim3(threads), 0, stream, (const float*)table, tokens, x, D, V, scale);
    else if (table_dtype == MYNAH_BF16)
        mynah_launch(embed_gather_kernel<bf16>, dim3(T), dim3(threads), 0, stream, (const bf16*)table, tokens, x, D, V, scale);
    else
        return mynah_fail("embed_gather: unsupported table dtype %d", table_dtype);
    return mynah_check_launch("embed_gather");
}

// x[t, :] = E[token_t, :] + P[row_t, :] with row_t = (token before * mul_prev + token_t * mul_cur) mod buckets, and row_t =
// buckets for a sequence's first token. The token before is the row above, or, for the first row of a sequence's piece, what
// the sequence's last step left in last_token[slot]; that row's CTA then leaves the piece's last token there (no other CTA
// touches the entry, so the read and the write are ordered inside one thread).
template <typename TW>
__global__ void embed_pairs_kernel(const TW* __restrict__ table, const TW* __restrict__ pairs, const int* __restrict__ tokens,
                                   const int* __restrict__ tok_seq, const int* __restrict__ tok_pos, const int* __restrict__ cu_q,
                                   const int* __restrict__ slots, int* __restrict__ last_token, float* __restrict__ x, int D, int V,
                                   int n_slots, int buckets, long long mul_prev, long long mul_cur, int* __restrict__ status) {
    __shared__ int row_s;
    griddep_launch_small();
    griddep_wait();
    const int t = blockIdx.x, b = tok_seq[t];
    float* out = x + (size_t)t * D;
    const int tok = tokens[t];
    if (b < 0 || tok < 0 || tok >= V) {      // a padding row (or an id that the host refuses already)
        for (int i = threadIdx.x; i < D; i += blockDim.x) out[i] = 0.f;
        return;
    }
    if (threadIdx.x == 0) {
        const int slot = slots[b], q0 = cu_q[b];
        const bool live = slot >= 0 && slot < n_slots;
        int before = t > q0 ? tokens[t - 1] : (live ? last_token[slot] : 0);
        if (t == q0 && live) last_token[slot] = tokens[cu_q[b + 1] - 1];
        int row = buckets;
        if (tok_pos[t] > 0) {
            if (before < 0 || before >= V) {
                atomicOr(status, MYNAH_ST_TOKEN_RANGE);
                before = 0;
            }
            // both products reduced before they are added: no overflow for any ids and multipliers of 31 bits
            row = (int)(((long long)before * mul_prev % buckets + (long long)tok * mul_cur % buckets) % buckets);
        }
        row_s = row;
    }
    __syncthreads();
    const TW* er = table + (size_t)tok * D;
    const TW* pr = pairs + (size_t)row_s * D;
    for (int i = threadIdx.x; i < D; i += blockDim.x) out[i] = to_f32(er[i]) + to_f32(pr[i]);
}

// table [V][D], pairs [buckets + 1][D], both in table_dtype; last_token int32 [n_slots + 1], kept from step to step.
MYNAH_API int mynah_embed_pairs(const void* table, const void* pairs, int table_dtype, const int* tokens, const int* tok_seq, const int* tok_pos,
                                const int* cu_q, const int* slots, int* last_token, float* x, int T, int D, int V, int n_slots, int buckets,
                                long long mul_prev, long long mul_cur, int* status, cudaStream_t stream) {
    if (T == 0) return 0;
    MYNAH_REQUIRE(T > 0 && D > 0 && V > 0 && buckets > 0, "embed_pairs: bad sizes T=%d D=%d V=%d buckets=%d", T, D, V, buckets);
    MYNAH_REQUIRE(mul_prev >= 0 && mul_cur >= 0 && mul_prev < (1ll << 31) && mul_cur < (1ll << 31), "embed_pairs: the multipliers must lie in 0 .. 2^31 - 1");
    const int threads = D >= 1024 ? 256 : (D >= 256 ? 128 : 64);
    if (table_dtype == MYNAH_F32)
        mynah_launch(embed_pairs_kernel<float>, dim3(T), dim3(threads), 0, stream, (const float*)table, (const float*)pairs, tokens, tok_seq, tok_pos,
                     cu_q, slots, last_token, x, D, V, n_slots, buckets, mul_prev, mul_cur, status);
    else if (table_dtype == MYNAH_BF16)
        mynah_launch(embed_pairs_kernel<bf16>, dim3(T), dim3(threads), 0, stream, (const bf16*)table, (const bf16*)pairs, tokens, tok_seq, tok_pos,
                     cu_q, slots, last_token, x, D, V, n_slots, buckets, mul_prev, mul_cur, status);
    else
        return mynah_fail("embed_pairs: unsupported table dtype %d", table_dtype);
    return mynah_check_launch("embed_pairs");
}

// --------------------------------------------------------------- RMSNorm
// v = x[r] (+ dscale * delta[r]);  x[r] = v when delta is given and every row is taken (no `rows`);
// out[i] = (v * s) * w   with   s = 1 / sqrt(mean(v^2) + eps)
// (mynah-slm src/kernels.c:118-128; plain gain, not 1+w). `rows`, when given,
// selects the rows to normalise (the rows whose logits are wanted); out then
// has one row per selected row.
template <typename TA>
__global__ void rmsnorm_kernel(float* __restrict__ x, const TA* __restrict__ delta, VecRef w,
                               const int* __restrict__ rows, TA* __restrict__ out, int D, float eps, float dscale) {
    __shared__ float red[32];
    griddep_launch_small();
    griddep_wait();
    const int r = rows ? rows[blockIdx.x] : blockIdx.x;
    float* xr = x + (size_t)r * D;
    const TA* dr = delta ? delta + (size_t)r * D : nullptr;
    // the sum is kept in x when every row is normalised once; selected rows may repeat (several CTAs on one
    // row), so with a selection x is only read
    const bool keep = dr != nullptr && rows == nullptr;
    float ss = 0.f;
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        float v = xr[i];
        if (dr) {
            v += to_f32(dr[i]) * dscale;
            if (keep) xr[i] = v;
        }
        ss += v * v;
    }
    ss = block_sum(ss, red);
    const float s = 1.0f / sqrtf(ss / (float)D + eps);
    TA* o = out + (size_t)blockIdx.x * D;
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        float v = xr[i];
        if (dr && !keep) v += to_f32(dr[i]) * dscale;
        o[i] = from_f32<TA>((v * s) * w.at(i));
    }
}

// The same norm with the row kept in registers: four consecutive elements per thread, one pass over
// memory. Taken when D is a multiple of 4 and fits (D <= 4 * 1024).
template <typename TA>
__global__ void rmsnorm_vec4_kernel(float* __restrict__ x, const TA* __restrict__ delta, VecRef w,
                                    const int* __restrict__ rows, TA* __restrict__ out, int D, float eps, float dscale) {
    __shared__ float red[32];
    griddep_launch_small();
    griddep_wait();
    const int r = rows ? rows[blockIdx.x] : blockIdx.x;
    float* xr = x + (size_t)r * D;
    const int i = threadIdx.x * 4;
    const bool on = i < D;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on) {
        v = *reinterpret_cast<const float4*>(xr + i);
        if (delta) {
            const TA* dr = delta + (size_t)r * D + i;
            v.x += to_f32(dr[0]) * dscale; v.y += to_f32(dr[1]) * dscale; v.z += to_f32(dr[2]) * dscale; v.w += to_f32(dr[3]) * dscale;
            if (rows == nullptr) *reinterpret_cast<float4*>(xr + i) = v;     // (selected rows may repeat: x is only read)
        }
    }
    float ss = (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
    ss = block_sum(ss, red);
    const float s = 1.0f / sqrtf(ss / (float)D + eps);
    if (on) {
        TA* o = out + (size_t)blockIdx.x * D + i;
        o[0] = from_f32<TA>((v.x * s) * w.at(i));
        o[1] = from_f32<TA>((v.y * s) * w.at(i + 1));
        o[2] = from_f32<TA>((v.z * s) * w.at(i + 2));
        o[3] = from_f32<TA>((v.w * s) * w.at(i + 3));
    }
}

// Eight consecutive elements per thread: the row, the pending delta, the gains and the result all move as 16-byte
// vectors. Taken when D is a multiple of 8 and fits (D <= 8 * 1024), for any number of rows, so that a row's sum
// has the same order in every step.
template <typename TA>
__global__ void rmsnorm_vec8_kernel(float* __restrict__ x, const TA* __restrict__ delta, VecRef w,
                                    const int* __restrict__ rows, TA* __restrict__ out, int D, float eps, float dscale) {
    __shared__ float red[32];
    griddep_launch_small();
    griddep_wait();
    const int r = rows ? rows[blockIdx.x] : blockIdx.x;
    float* xr = x + (size_t)r * D;
    const int i = threadIdx.x * 8;
    const bool on = i < D;
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (on) {
        load8(xr + i, v);
        if (delta) {
            float d[8];
            load8(delta + (size_t)r * D + i, d);
#pragma unroll
            for (int j = 0; j < 8; j++) v[j] += d[j] * dscale;
            if (rows == nullptr) store8(xr + i, v);        // (selected rows may repeat: x is only read)
        }
    }
    float ss = ((v[0] * v[0] + v[1] * v[1]) + (v[2] * v[2] + v[3] * v[3])) + ((v[4] * v[4] + v[5] * v[5]) + (v[6] * v[6] + v[7] * v[7]));
    ss = block_sum(ss, red);
    const float s = 1.0f / sqrtf(ss / (float)D + eps);
    if (on) {
        float g[8];
        load_gain8(w, i, g);
#pragma unroll
        for (int j = 0; j < 8; j++) v[j] = (v[j] * s) * g[j];
        store8(out + (size_t)blockIdx.x * D + i, v);
    }
}

MYNAH_API int mynah_rmsnorm(float* x, const void* delta, const void* w, int w_dtype, const int* rows,
                            void* out, int act_dtype, int n_rows, int D, float eps, float dscale, cudaStream_t stream) {
    if (n_rows == 0) return 0;
    MYNAH_REQUIRE(n_rows > 0 && D > 0, "rmsnorm: bad sizes rows=%d D=%d", n_rows, D);
    MYNAH_REQUIRE(w_dtype == MYNAH_F32 || w_dtype == MYNAH_BF16, "rmsnorm: unsupported gain dtype %d", w_dtype);
    const VecRef wr{w, w_dtype};
    const bool aligned16 = (((uintptr_t)x | (uintptr_t)delta | (uintptr_t)w | (uintptr_t)out) & 15) == 0;
    if (D % 8 == 0 && D <= 8192 && D >= 256 && aligned16) {
        const int threads = ((D / 8 + 31) / 32) * 32;
        if (act_dtype == MYNAH_F32)
            mynah_launch(rmsnorm_vec8_kernel<float>, dim3(n_rows), dim3(threads), 0, stream, x, (const float*)delta, wr, rows, (float*)out, D, eps, dscale);
        else if (act_dtype == MYNAH_BF16)
            mynah_launch(rmsnorm_vec8_kernel<bf16>, dim3(n_rows), dim3(threads), 0, stream, x, (const bf16*)delta, wr, rows, (bf16*)out, D, eps, dscale);
        else
            return mynah_fail("rmsnorm: unsupported activation dtype %d", act_dtype);
        return mynah_check_launch("rmsnorm");
    }
    if (D % 4 == 0 && D <= 4096 && D >= 128) {
        const int threads = ((D / 4 + 31) / 32) * 32;
        if (act_dtype == MYNAH_F32)
            mynah_launch(rmsnorm_vec4_kernel<float>, dim3(n_rows), dim3(threads), 0, stream, x, (const float*)delta, wr, rows, (float*)out, D, eps, dscale);
        else if (act_dtype == MYNAH_BF16)
            mynah_launch(rmsnorm_vec4_kernel<bf16>, dim3(n_rows), dim3(threads), 0, stream, x, (const bf16*)delta, wr, rows, (bf16*)out, D, eps, dscale);
        else
            return mynah_fail("rmsnorm: unsupported activation dtype %d", act_dtype);
        return mynah_check_launch("rmsnorm");
    }
    const int threads = D >= 2048 ? 512 : (D >= 512 ? 256 : (D >= 128 ? 128 : 32));
    if (act_dtype == MYNAH_F32)
        mynah_launch(rmsnorm_kernel<float>, dim3(n_rows), dim3(threads), 0, stream, x, (const float*)delta, wr, rows, (float*)out, D, eps, dscale);
    else if (act_dtype == MYNAH_BF16)
        mynah_launch(rmsnorm_kernel<bf16>, dim3(n_rows), dim3(threads), 0, stream, x, (const bf16*)delta, wr, rows, (bf16*)out, D, eps, dscale);
    else
        return mynah_fail("rmsnorm: unsupported activation dtype %d", act_dtype);
    return mynah_check_launch("rmsnorm");
}

// ----------------------------------------------------------- residual add
template <typename TA>
__global__ void residual_add_kernel(float* __restrict__ x, const TA* __restrict__ delta, size_t n, float scale) {
    griddep_launch();
    griddep_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] += to_f32(delta[i]) * scale;  // mynah-slm src/kernels.c:222-224 (scale 1 there)
}

MYNAH_API int mynah_residual_add(float* x, const void* delta, int act_dtype, long long n, float scale, cudaStream_t stream) {
    if (n == 0) return 0;
    const unsigned blocks = (unsigned)ceil_div_ll(n, 256);
    if (act_dtype == MYNAH_F32)
        mynah_launch(residual_add_kernel<float>, dim3(blocks), dim3(256), 0, stream, x, (const float*)delta, (size_t)n, scale);
    else if (act_dtype == MYNAH_BF16)
        mynah_launch(residual_add_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, x, (const bf16*)delta, (size_t)n, scale);
    else
        return mynah_fail("residual_add: unsupported activation dtype %d", act_dtype);
    return mynah_check_launch("residual_add");
}

// x[t][:] += v[:] for every row: one learned vector added to the whole stream (fp32).
__global__ void residual_add_row_kernel(float* __restrict__ x, const float* __restrict__ v, size_t n, int D) {
    griddep_launch();
    griddep_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] += v[i % D];
}

MYNAH_API int mynah_residual_add_row(float* x, const float* v, long long n_rows, int D, cudaStream_t stream) {
    if (n_rows == 0) return 0;
    MYNAH_REQUIRE(n_rows > 0 && D > 0, "residual_add_row: bad sizes");
    const long long n = n_rows * D;
    mynah_launch(residual_add_row_kernel, dim3((unsigned)ceil_div_ll(n, 256)), dim3(256), 0, stream, x, v, (size_t)n, D);
    return mynah_check_launch("residual_add_row");
}

// ----------------------------------------------------------------- SwiGLU
// a = (g * sigmoid(g)) * u with the sigmoid that never exponentiates a
// positive argument (mynah-slm src/kernels.c:193-205). gate_up is [T, 2F]:
// gate in columns [0, F), up in [F, 2F).
__device__ __forceinline__ float stable_sigmoid(float v) {
    // e^-|v| never overflows; the select keeps both branches of the reference's stable form exact
    const float e = expf(-fabsf(v));
    return (v >= 0.f ? 1.0f : e) / (1.0f + e);
}

template <typename TA>
__global__ void swiglu_kernel(const TA* __restrict__ gate_up, TA* __restrict__ out, int F) {
    griddep_launch();
    griddep_wait();
    const int t = blockIdx.x;
    const int i = blockIdx.y * blockDim.x + threadIdx.x;
    if (i >= F) return;
    const TA* row = gate_up + (size_t)t * 2 * F;
    const float g = to_f32(row[i]), u = to_f32(row[F + i]);
    out[(size_t)t * F + i] = from_f32<TA>((g * stable_sigmoid(g)) * u);
}

// Eight elements per thread (16-byte loads and stores) when F is a multiple of 8.
template <typename TA>
__global__ void swiglu_vec8_kernel(const TA* __restrict__ gate_up, TA* __restrict__ out, int F) {
    griddep_launch();
    griddep_wait();
    const int t = blockIdx.x;
    const int i = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
    if (i >= F) return;
    const TA* row = gate_up + (size_t)t * 2 * F;
    float g[8], u[8], o[8];
    load8(row + i, g);
    load8(row + F + i, u);
#pragma unroll
    for (int j = 0; j < 8; j++) o[j] = (g[j] * stable_sigmoid(g[j])) * u[j];
    store8(out + (size_t)t * F + i, o);
}

MYNAH_API int mynah_swiglu(const void* gate_up, void* out, int act_dtype, int T, int F, cudaStream_t stream) {
    if (T == 0) return 0;
    MYNAH_REQUIRE(T > 0 && F > 0, "swiglu: bad sizes T=%d F=%d", T, F);
    MYNAH_REQUIRE(ceil_div(F, 256) <= 65535, "swiglu: width %d exceeds one launch", F);
    if (F % 8 == 0) {
        const dim3 vgrid(T, ceil_div(F / 8, 128));
        if (act_dtype == MYNAH_F32)
            mynah_launch(swiglu_vec8_kernel<float>, vgrid, dim3(128), 0, stream, (const float*)gate_up, (float*)out, F);
        else if (act_dtype == MYNAH_BF16)
            mynah_launch(swiglu_vec8_kernel<bf16>, vgrid, dim3(128), 0, stream, (const bf16*)gate_up, (bf16*)out, F);
        else
            return mynah_fail("swiglu: unsupported activation dtype %d", act_dtype);
        return mynah_check_launch("swiglu");
    }
    const dim3 grid(T, ceil_div(F, 256));
    if (act_dtype == MYNAH_F32)
        mynah_launch(swiglu_kernel<float>, dim3(grid), dim3(256), 0, stream, (const float*)gate_up, (float*)out, F);
    else if (act_dtype == MYNAH_BF16)
        mynah_launch(swiglu_kernel<bf16>, dim3(grid), dim3(256), 0, stream, (const bf16*)gate_up, (bf16*)out, F);
    else
        return mynah_fail("swiglu: unsupported activation dtype %d", act_dtype);
    return mynah_check_launch("swiglu");
}

// ------------------------------------------------- embedding with learned positions
// x[t, :] = E[token_t, :] + P[position_t, :]        (neither scaled); fp32 sum of the two stored rows
template <typename TW>
__global__ void embed_positions_kernel(const TW* __restrict__ table, const TW* __restrict__ pos_table,
                                       const int* __restrict__ tokens, const int* __restrict__ tok_pos,
                                       float* __restrict__ x, int D, int V, int n_pos, int* __restrict__ status) {
    griddep_launch();
    griddep_wait();
    const int t = blockIdx.x;
    const int tok = tokens[t], pos = tok_pos[t];
    float* out = x + (size_t)t * D;
    const bool bad_tok = tok < 0 || tok >= V, bad_pos = pos < 0 || pos >= n_pos;
    if (bad_tok || bad_pos) {
        if (threadIdx.x == 0) atomicOr(status, bad_tok ? 4 : 2);      // token / position outside its table
        for (int i = threadIdx.x; i < D; i += blockDim.x) out[i] = 0.f;
        return;
    }
    const TW* row = table + (size_t)tok * D;
    const TW* prow = pos_table + (size_t)pos * D;
    for (int i = threadIdx.x; i < D; i += blockDim.x) out[i] = to_f32(row[i]) + to_f32(prow[i]);
}

MYNAH_API int mynah_embed_positions(const void* table, const void* pos_table, int table_dtype, const int* tokens,
                                    const int* tok_pos, float* x, int T, int D, int V, int n_pos, int* status,
                                    cudaStream_t stream) {
    if (T == 0) return 0;
    MYNAH_REQUIRE(T > 0 && D > 0 && V > 0 && n_pos > 0, "embed_positions: bad sizes T=%d D=%d V=%d positions=%d", T, D, V, n_pos);
    const int threads = D >= 1024 ? 256 : (D >= 256 ? 128 : 64);
    if (table_dtype == MYNAH_F32)
        mynah_launch(embed_positions_kernel<float>, dim3(T), dim3(threads), 0, stream, (const float*)table,
                     (const float*)pos_table, tokens, tok_pos, x, D, V, n_pos, status);
    else if (table_dtype == MYNAH_BF16)
        mynah_launch(embed_positions_kernel<bf16>, dim3(T), dim3(threads), 0, stream, (const bf16*)table,
                     (const bf16*)pos_table, tokens, tok_pos, x, D, V, n_pos, status);
    else
        return mynah_fail("embed_positions: unsupported table dtype %d", table_dtype);
    return mynah_check_launch("embed_positions");
}

// ------------------------------------------------------------ activations
// In place or not: out[i] = act(in[i]), computed in fp32. 0: gelu with erf, 0.5 z (1 + erf(z / sqrt 2));
// 1: gelu with tanh, 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))); 2: silu; 3: relu; 4: the square of relu.
__device__ __forceinline__ float act_apply(float z, int act) {
    switch (act) {
        case 0: return 0.5f * z * (1.0f + erff(z * 0.70710678118654752440f));
        case 1: return 0.5f * z * (1.0f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z)));
        case 2: return z / (1.0f + expf(-z));
        case 3: return fmaxf(z, 0.f);
        default: { const float r = fmaxf(z, 0.f); return r * r; }
    }
}

template <typename T>
__global__ void activation_kernel(const T* __restrict__ in, T* __restrict__ out, long long n, int act) {
    griddep_launch_small();
    griddep_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = from_f32<T>(act_apply(to_f32(in[i]), act));
}

// eight consecutive elements a thread, 16-byte vectors
template <typename T>
__global__ void activation8_kernel(const T* __restrict__ in, T* __restrict__ out, long long n8, int act) {
    griddep_launch_small();
    griddep_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n8) return;
    float v[8];
    load8(in + i * 8, v);
#pragma unroll
    for (int k = 0; k < 8; k++) v[k] = act_apply(v[k], act);
    store8(out + i * 8, v);
}

MYNAH_API int mynah_activation(const void* in, void* out, int dtype, long long n, int act, cudaStream_t stream) {
    if (n == 0) return 0;
    MYNAH_REQUIRE(n > 0 && act >= 0 && act <= 4, "activation: bad arguments n=%lld act=%d", n, act);
    if (n % 8 == 0 && ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(out)) & 31) == 0 &&
        (dtype == MYNAH_F32 || dtype == MYNAH_BF16)) {
        const long long n8 = n / 8;
        const unsigned blocks8 = (unsigned)ceil_div_ll(n8, 256);
        if (dtype == MYNAH_F32)
            mynah_launch(activation8_kernel<float>, dim3(blocks8), dim3(256), 0, stream, (const float*)in, (float*)out, n8, act);
        else
            mynah_launch(activation8_kernel<bf16>, dim3(blocks8), dim3(256), 0, stream, (const bf16*)in, (bf16*)out, n8, act);
        return mynah_check_launch("activation");
    }
    const unsigned blocks = (unsigned)ceil_div_ll(n, 256);
    if (dtype == MYNAH_F32)
        mynah_launch(activation_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float*)in, (float*)out, n, act);
    else if (dtype == MYNAH_BF16)
        mynah_launch(activation_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, (const bf16*)in, (bf16*)out, n, act);
    else
        return mynah_fail("activation: unsupported dtype %d", dtype);
    return mynah_check_launch("activation");
}

// ------------------------------------------------------------------ cast
// out[i] = in[i] rounded to the activation type: what a sublayer reads of the fp32 residual stream when no
// norm stands in front of it.
template <typename T>
__global__ void cast_f32_kernel(const float* __restrict__ in, T* __restrict__ out, long long n) {
    griddep_launch_small();
    griddep_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = from_f32<T>(in[i]);
}

MYNAH_API int mynah_cast_f32(const float* in, void* out, int out_dtype, long long n, cudaStream_t stream) {
    if (n == 0) return 0;
    MYNAH_REQUIRE(n > 0, "cast_f32: bad size %lld", n);
    const unsigned blocks = (unsigned)ceil_div_ll(n, 256);
    if (out_dtype == MYNAH_BF16)
        mynah_launch(cast_f32_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, in, (bf16*)out, n);
    else if (out_dtype == MYNAH_F32)
        mynah_launch(cast_f32_kernel<float>, dim3(blocks), dim3(256), 0, stream, in, (float*)out, n);
    else
        return mynah_fail("cast_f32: unsupported dtype %d", out_dtype);
    return mynah_check_launch("cast_f32");
}

// ----------------------------------------------------------------- scale
// x[i] *= s in place (fp32): a head whose logits are multiplied by a constant.
// four values a thread, in one 16-byte access where they are aligned
__global__ void scale_f32_kernel(float* __restrict__ x, long long n, float s) {
    griddep_launch_small();
    griddep_wait();
    const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (i + 3 < n && (reinterpret_cast<uintptr_t>(x) & 15) == 0) {
        float4 v = *reinterpret_cast<const float4*>(x + i);
        v.x *= s; v.y *= s; v.z *= s; v.w *= s;
        *reinterpret_cast<float4*>(x + i) = v;
        return;
    }
    for (long long j = i; j < n && j < i + 4; j++) x[j] *= s;
}

// x[i] = c tanh(x[i] / c) in place (fp32): a head whose logits are capped.
__global__ void softcap_f32_kernel(float* __restrict__ x, long long n, float c, float inv_c) {
    griddep_launch_small();
    griddep_wait();
    const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (i + 3 < n) {
        float4 v = *reinterpret_cast<const float4*>(x + i);
        v.x = c * tanhf(v.x * inv_c);
        v.y = c * tanhf(v.y * inv_c);
        v.z = c * tanhf(v.z * inv_c);
        v.w = c * tanhf(v.w * inv_c);
        *reinterpret_cast<float4*>(x + i) = v;
    } else {
        for (long long j = i; j < n; j++) x[j] = c * tanhf(x[j] * inv_c);
    }
}

MYNAH_API int mynah_softcap_f32(float* x, long long n, float c, cudaStream_t stream) {
    if (n == 0) return 0;
    MYNAH_REQUIRE(n > 0 && c > 0.f && ((uintptr_t)x & 15) == 0, "softcap_f32: bad size %lld, cap or alignment", n);
    mynah_launch(softcap_f32_kernel, dim3((unsigned)ceil_div_ll(ceil_div_ll(n, 4), 256)), dim3(256), 0, stream, x, n, c, 1.0f / c);
    return mynah_check_launch("softcap_f32");
}

MYNAH_API int mynah_scale_f32(float* x, long long n, float s, cudaStream_t stream) {
    if (n == 0) return 0;
    MYNAH_REQUIRE(n > 0, "scale_f32: bad size %lld", n);
    mynah_launch(scale_f32_kernel, dim3((unsigned)ceil_div_ll(n, 1024)), dim3(256), 0, stream, x, n, s);
    return mynah_check_launch("scale_f32");
}
