// Linear attention with decays, in three kinds. Per head, with S [dim x vd] the state (fp32, per slot) and
// k, q, v the token's rows (q times q_scale):
//
//   GLA     S_t = diag(a_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   a_t = sigmoid(z_t)^(1/tau) a key channel,
//           z_t = W_2 r_t + b  (r_t: the token's narrow row of `rank` values)
//   MLSTM   (the matrix memory of xLSTM) log gates i = cap tanh((p_i + b_i)/cap), f = log sigmoid(cap tanh((p_f + b_f)/cap));
//           m_t = max(f + m_(t-1), i)  (from m = 0);  S and n decay by exp(f + m_(t-1) - m_t) and take exp(i - m_t) k v^T
//           (n: the same with k alone);   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
//   FIXED   (retention) S_t = decay_head S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
//
// and behind either, in the same kernel:  out = o / sqrt(mean(o^2) + eps) * w[head, column] * act(gate),  act silu (GLA, FIXED)
// or sigmoid (MLSTM), written in the rows' type to `out`'s columns [o_off + head * vd, ...).
//
// Token form (gm_token): a CTA takes a head of a sequence and walks its tokens; a thread owns fixed entries of S. One token a
// sequence (a decode step): S passes once through registers, from memory and back. Several: S stays in shared memory where it
// fits. All arithmetic fp32; the only form of the 32-bit run.
//
// Chunk form, for bfloat16 prompts, chunks of 64 tokens, three kernels of which only the middle one follows the sequence:
//
//   gm_chunk_state   a chunk's own contribution to the state, U = sum_s diag(decay from s to the chunk's end) k_s v_s^T, all
//                    chunks side by side; GLA also makes z (a small product), the log decays and their running sums b
//   gm_chunk_scan    S before every chunk, elementwise in chunk order, in place over U; the sequence's state at the end
//   gm_chunk_out     a chunk's outputs from the state before it and its own scores, then norm and gate
//
// With b_t the running sum of log decays inside the chunk (kept as binary logarithms, so e^ is 2^ in the kernels): o_t = sum_{s<=t} <q_t e^{b_t}, k_s e^{-b_s}> v_s + (q_t e^{b_t}) S_0.
// GLA scales q and k around half the chunk's total per channel (exponents stay within half the total), and where a chunk's
// total exceeds GLA_RANGE forms every score channel by channel instead (all exponents then <= 0). MLSTM needs no scaling of q
// and k: with g_s = i_s - F_s and M_t = max(m_0, max_{s<=t} g_s), m_t = F_t + M_t, a score counts e^{g_s - M_t} and the old
// state e^{m_0 - M_t}. FIXED needs none of this: a score counts decay^(t - s), the old state decay^(t + 1), both as 2^ of the
// head's binary logarithm.
//
// The products run on mma.sync (bf16 in, fp32 out). q, k and v of the MLSTM and of FIXED and v of the GLA are bfloat16 as projected; every
// fp32 operand (scaled q and k, scores, the state) is carried as a sum of two bfloat16 values, which leaves a relative error
// of about 2^-17 in it.
#include "layout.cuh"
#include "mma_frag.cuh"

namespace {

using namespace mmafrag;

enum GmKind : int { GLA = 0, MLSTM = 1, FIXED = 2 };

constexpr int GC = 64;                  // tokens of a chunk
constexpr int G_THREADS = 256;
constexpr float GLA_RANGE = 86.f;       // total of binary log decays (of one channel, over a chunk) up to which q and k are scaled
constexpr float LOG2E = 1.4426950408889634f;
constexpr float MLSTM_FLOOR = 1e-6f;

struct GmArgs {
    int B, H, dim, vd, ld, ldo, o_off;
    int q_off, k_off, v_off, g_off;     // first columns of q, k, v and the gate in the rows
    int a_off, b_off;                   // GLA: the narrow rows; MLSTM: the input gates and the forget gates (H values each)
    int rank, n_slots;
    float q_scale, inv_tau, cap, eps;
};

// What a sequence's head carries: S [dim][vd]; MLSTM also n [dim] and m.
struct GmState {
    float *S, *n, *m;                   // [slots + 1][H][...]
};

__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
// log2(sigmoid(z)): the logarithm of 1 + 2^-|.| from the hardware's log2 (absolute error about 2^-22), by its series where the
// summand is small, so that decays next to one keep their relative accuracy
__device__ __forceinline__ float log2_sigmoid(float z) {
    const float y = z * LOG2E, e = exp2f(-fabsf(y));
    const float s = e < 0.015625f ? e * fmaf(e, fmaf(e, fmaf(e, -0.25f, 0.33333334f), -0.5f), 1.0f) * LOG2E : __log2f(1.0f + e);
    return fminf(y, 0.f) - s;
}
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
template <int KIND> __device__ __forceinline__ float gate_act(float z) { return KIND == MLSTM ? sigmoid_f(z) : z * sigmoid_f(z); }

// ------------------------------------------------------------------------------------------------ token form
constexpr int TOK_BATCH = 8;            // rows of S a thread has in flight

template <int VEC> struct Vec;
template <> struct Vec<1> { typedef float type; };
template <> struct Vec<4> { typedef float4 type; };
__device__ __forceinline__ void unpack(float v, float (&x)[1]) { x[0] = v; }
__device__ __forceinline__ void unpack(const float4& v, float (&x)[4]) { x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w; }
__device__ __forceinline__ float repack(const float (&x)[1]) { return x[0]; }
__device__ __forceinline__ float4 repack(const float (&x)[4]) { return make_float4(x[0], x[1], x[2], x[3]); }

// grid (H, B). `in_smem`: S is copied to shared memory first (several tokens), else it is updated where it lies.
template <typename T, int KIND, int VEC>
__global__ void __launch_bounds__(512)
gm_token_kernel(const T* __restrict__ p, const T* __restrict__ w2, const float* __restrict__ bias, const float* __restrict__ w_norm,
                GmState st, T* __restrict__ out, const int* __restrict__ cu_q, const int* __restrict__ slots, GmArgs a, int in_smem) {
    typedef typename Vec<VEC>::type V;
    extern __shared__ __align__(16) float sm[];
    griddep_wait();
    const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, NT = blockDim.x;
    const int slot = slots[b], q0 = cu_q[b], q1 = cu_q[b + 1];
    if (slot < 0 || slot >= a.n_slots || q1 <= q0) return;
    const int dim = a.dim, vd = a.vd;
    const int cols = vd / VEC, groups = NT / cols;             // threads a row of S, rows at a time
    const int col = tid % cols, grp = tid / cols;
    const bool on = grp < groups;
    float* qs = sm;                                            // [dim]
    float* ks = qs + dim;                                      // [dim]
    float* as = ks + dim;                                      // [dim]: decay of the channel
    float* vs = as + dim;                                      // [vd]
    float* rs = vs + vd;                                       // [rank] the narrow row (GLA)
    float* os = rs + a.rank;                                   // [vd]
    float* red32 = os + vd;                                    // [32]
    float* red = reinterpret_cast<float*>((reinterpret_cast<uintptr_t>(red32 + 32) + 15) & ~(uintptr_t)15);   // [groups][vd]
    float* ns = red + (size_t)groups * vd;                     // [dim] (MLSTM)
    float* Ss = reinterpret_cast<float*>((reinterpret_cast<uintptr_t>(ns + dim) + 15) & ~(uintptr_t)15);      // [dim][vd]
    __shared__ float keep_s, add_s, m_s;
    const size_t sh = (size_t)slot * a.H + h;
    float* Sg = st.S + sh * dim * vd;
    float* Sp = Sg;
    if (in_smem) {
        for (int e = tid; e < dim * vd; e += NT) Ss[e] = Sg[e];
        Sp = Ss;
    }
    if (KIND == MLSTM) {
        for (int c = tid; c < dim; c += NT) ns[c] = st.n[sh * dim + c];
        if (tid == 0) m_s = st.m[sh];
    }
    V* Sv = reinterpret_cast<V*>(Sp);
    // one token: the first rows of S are on their way while the token's rows are prepared
    V first[TOK_BATCH];
    if (!in_smem && on) {
#pragma unroll
        for (int i = 0; i < TOK_BATCH; i++) {
            const int r = grp + i * groups;
            if (r < dim) first[i] = Sv[(size_t)r * cols + col];
        }
    }
    for (int t = q0; t < q1; t++) {
        const T* row = p + (size_t)t * a.ld;
        // the first column's gate and weight are on their way while the token is worked on
        const float z_first = tid < vd ? to_f32(row[a.g_off + h * vd + tid]) : 0.f, w_first = tid < vd ? w_norm[h * vd + tid] : 0.f;
        __syncthreads();                                       // the token before is done (and m, n, S are in place)
        for (int c = tid; c < dim; c += NT) {
            qs[c] = to_f32(row[a.q_off + h * dim + c]) * a.q_scale;
            ks[c] = to_f32(row[a.k_off + h * dim + c]);
        }
        for (int c = tid; c < vd; c += NT) vs[c] = to_f32(row[a.v_off + h * vd + c]);
        if (KIND == GLA) {
            for (int c = tid; c < a.rank; c += NT) rs[c] = to_f32(row[a.a_off + c]);
            // the thread's row of W_2, too (up to 16 values; the first token of a step brings it from memory)
            const bool short_row = a.rank <= 16 && (a.rank * sizeof(T)) % 32 == 0;
            float w_row[16], b_first = 0.f;
            if (tid < dim) {
                b_first = bias[h * dim + tid];
                if (short_row) {
                    const T* w = w2 + (size_t)(h * dim + tid) * a.rank;
#pragma unroll
                    for (int r = 0; r < 16; r += 8)
                        if (r < a.rank) load8(w + r, *reinterpret_cast<float(*)[8]>(w_row + r));
                }
            }
            __syncthreads();
            for (int c = tid; c < dim; c += NT) {
                const T* w = w2 + (size_t)(h * dim + c) * a.rank;
                float z = 0.f;
                if (c == tid && short_row) {
#pragma unroll
                    for (int r = 0; r < 16; r++)
                        if (r < a.rank) z = fmaf(w_row[r], rs[r], z);
                } else if ((a.rank * sizeof(T)) % 32 == 0) {              // rows of whole 32-byte groups: 8 values a load
                    for (int r = 0; r < a.rank; r += 8) {
                        float wv[8];
                        load8(w + r, wv);
#pragma unroll
                        for (int j = 0; j < 8; j++) z = fmaf(wv[j], rs[r + j], z);
                    }
                } else {
                    for (int r = 0; r < a.rank; r++) z = fmaf(to_f32(w[r]), rs[r], z);
                }
                as[c] = expf(log_sigmoid_f(z + (c == tid ? b_first : bias[h * dim + c])) * a.inv_tau);
            }
        } else if (KIND == MLSTM && tid == 0) {
            const float i = a.cap * tanhf((to_f32(row[a.a_off + h]) + bias[h]) / a.cap);
            const float f = log_sigmoid_f(a.cap * tanhf((to_f32(row[a.b_off + h]) + bias[a.H + h]) / a.cap));
            const float m_new = fmaxf(f + m_s, i);
            keep_s = expf(f + m_s - m_new);
            add_s = expf(i - m_new);
            m_s = m_new;
        }
        __syncthreads();
        const float keep = KIND == MLSTM ? keep_s : (KIND == FIXED ? bias[h] : 0.f), add = KIND == MLSTM ? add_s : 1.f;
        float acc[VEC];
#pragma unroll
        for (int j = 0; j < VEC; j++) acc[j] = 0.f;
        if (on) {
            float vv[VEC];
#pragma unroll
            for (int j = 0; j < VEC; j++) vv[j] = vs[col * VEC + j] * add;
            for (int r0 = grp; r0 < dim; r0 += TOK_BATCH * groups) {
                V s[TOK_BATCH];
#pragma unroll
                for (int i = 0; i < TOK_BATCH; i++) {
                    const int r = r0 + i * groups;
                    if (r < dim) s[i] = (!in_smem && r0 == grp && t == q0) ? first[i] : Sv[(size_t)r * cols + col];
                }
#pragma unroll
                for (int i = 0; i < TOK_BATCH; i++) {
                    const int r = r0 + i * groups;
                    if (r < dim) {
                        float x[VEC];
                        unpack(s[i], x);
                        const float g = KIND == GLA ? as[r] : keep, kk = ks[r], qq = qs[r];
#pragma unroll
                        for (int j = 0; j < VEC; j++) {
                            x[j] = fmaf(kk, vv[j], g * x[j]);
                            acc[j] = fmaf(x[j], qq, acc[j]);
                        }
                        Sv[(size_t)r * cols + col] = repack(x);
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < VEC; j++) red[grp * vd + col * VEC + j] = acc[j];
        }
        float nq = 0.f;
        if (KIND == MLSTM) {
            for (int c = tid; c < dim; c += NT) {
                const float nn = fmaf(ks[c], add, keep * ns[c]);
                ns[c] = nn;
                nq = fmaf(nn, qs[c], nq);
            }
            nq = block_sum(nq, red32);                         // (synchronises)
        } else {
            __syncthreads();
        }
        const float inv_den = KIND == MLSTM ? 1.0f / (fmaxf(fabsf(nq), expf(-m_s)) + MLSTM_FLOOR) : 1.0f;
        if (KIND == MLSTM) __syncthreads();                    // red32 has been read; the partial sums are there
        float ss = 0.f;
        for (int c = tid; c < vd; c += NT) {
            float o = 0.f;
            for (int g = 0; g < groups; g++) o += red[g * vd + c];
            o *= inv_den;
            os[c] = o;
            ss = fmaf(o, o, ss);
        }
        const float r = 1.0f / sqrtf(block_sum(ss, red32) / (float)vd + a.eps);
        for (int c = tid; c < vd; c += NT) {
            const float z = c == tid ? z_first : to_f32(row[a.g_off + h * vd + c]), w = c == tid ? w_first : w_norm[h * vd + c];
            out[(size_t)t * a.ldo + a.o_off + h * vd + c] = from_f32<T>(os[c] * r * w * gate_act<KIND>(z));
        }
    }
    __syncthreads();
    if (in_smem)
        for (int e = tid; e < dim * vd; e += NT) Sg[e] = Ss[e];
    if (KIND == MLSTM) {
        for (int c = tid; c < dim; c += NT) st.n[sh * dim + c] = ns[c];
        if (tid == 0) st.m[sh] = m_s;
    }
}

// ------------------------------------------------------------------------------------------------ chunk form
// Scratch, per chunk number `flat` (find_query_tile's numbering) and head: U fp32 [dim][vd], then (MLSTM) un fp32 [dim], the
// chunk's (F total, own maximum) and the m before it; GLA: b fp32 [rows][H * dim], the running sums of log decays.
struct GmScratch {
    float *U, *un, *scal, *m0, *b;
};

__device__ __forceinline__ uint32_t hi_pack(float x, float y, float& rx, float& ry) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    rx = x - __bfloat162float(h.x);
    ry = y - __bfloat162float(h.y);
    return *reinterpret_cast<const uint32_t*>(&h);
}
// eight fp32 values as two bfloat16 summands each
__device__ __forceinline__ void split8(const float (&v)[8], uint4& hi, uint4& lo) {
    uint32_t hw[4], lw[4];
#pragma unroll
    for (int i = 0; i < 4; i++) {
        float rx, ry;
        hw[i] = hi_pack(v[2 * i], v[2 * i + 1], rx, ry);
        lw[i] = pack_bf16(rx, ry);
    }
    hi = make_uint4(hw[0], hw[1], hw[2], hw[3]);
    lo = make_uint4(lw[0], lw[1], lw[2], lw[3]);
}

// fragment addresses in a tile of rows `ld` bfloat16 apart
__device__ __forceinline__ uint32_t addr_a(uint32_t base, int ld, int r0, int k0, int lane) {       // A from [row][k]
    return base + (uint32_t)(((r0 + (lane & 7) + ((lane >> 3) & 1) * 8) * ld + k0 + (lane >> 4) * 8) * 2);
}
__device__ __forceinline__ uint32_t addr_at(uint32_t base, int ld, int k0, int m0, int lane) {      // A from [k][m], transposed load
    return base + (uint32_t)(((k0 + (lane & 7) + (lane >> 4) * 8) * ld + m0 + ((lane >> 3) & 1) * 8) * 2);
}
__device__ __forceinline__ uint32_t addr_b(uint32_t base, int ld, int n0, int k0, int lane) {       // B from [n][k]: two n-tiles
    return base + (uint32_t)(((n0 + (lane & 7) + (lane >> 4) * 8) * ld + k0 + ((lane >> 3) & 1) * 8) * 2);
}
__device__ __forceinline__ uint32_t addr_bt(uint32_t base, int ld, int k0, int n0, int lane) {      // B from [k][n], transposed load
    return base + (uint32_t)(((k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * ld + n0 + (lane >> 4) * 8) * 2);
}

// rows [0, nt) of `cols` values (a multiple of 8) into a tile of GC rows; the rest of the tile, up to colsP columns, is zero.
// The copies are asynchronous, one group: cp_async_wait and a barrier before the tile is read.
__device__ __forceinline__ void load_tile(bf16* dst, int ld, const bf16* __restrict__ src, size_t ld_src, int nt, int cols, int colsP) {
    const int ch = colsP / 8;
    for (int i = threadIdx.x; i < GC * ch; i += G_THREADS) {
        const int r = i / ch, c = (i % ch) * 8;
        const bool in = r < nt && c < cols;
        cp_async_16(smem_u32(dst + r * ld + c), in ? src + (size_t)r * ld_src + c : src, in);
    }
    cp_async_commit();
}
// four 8-value pieces of a thread, numbers i0, i0 + G_THREADS, ... of the tile's GC x (colsP / 8): loaded together
struct Pieces { int t[4], c[4]; bool in[4], on[4]; };
__device__ __forceinline__ Pieces pieces_of(int i0, int nt, int cols, int colsP) {
    Pieces p;
    const int ch = colsP / 8;
#pragma unroll
    for (int u = 0; u < 4; u++) {
        const int i = i0 + u * G_THREADS;
        p.t[u] = i / ch;
        p.c[u] = (i % ch) * 8;
        p.on[u] = i < GC * ch;
        p.in[u] = p.on[u] && p.t[u] < nt && p.c[u] < cols;
    }
    return p;
}
__device__ __forceinline__ void widen8(const uint4& u, float (&v)[8]) {
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; i++) {
        v[2 * i] = __uint_as_float(w[i] << 16);
        v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}

// MLSTM: F_t (running sums of the log forget gates) and g_t = i_t - F_t of a chunk, by warp 0; rows beyond nt: F of the last
// row, g = -inf. `gmax`: running maxima of g, or null.
__device__ __forceinline__ void mlstm_gates(const bf16* __restrict__ p, const float* __restrict__ bias, int t0, int nt, int h, const GmArgs& a,
                                            float* Fs, float* gs, float* gmax) {
    if (threadIdx.x >= 32) return;
    const int lane = threadIdx.x;
    float base = 0.f, mx = -INFINITY;
#pragma unroll
    for (int half = 0; half < GC / 32; half++) {
        const int t = half * 32 + lane;
        float f = 0.f, i = -INFINITY;
        if (t < nt) {
            const bf16* row = p + (size_t)(t0 + t) * a.ld;
            i = a.cap * tanhf((to_f32(row[a.a_off + h]) + bias[h]) / a.cap);
            f = log_sigmoid_f(a.cap * tanhf((to_f32(row[a.b_off + h]) + bias[a.H + h]) / a.cap));
        }
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, f, o);
            if (lane >= o) f += v;
        }
        f += base;
        base = __shfl_sync(0xffffffffu, f, 31);
        const float g = t < nt ? i - f : -INFINITY;
        Fs[t] = f;
        gs[t] = g;
        if (gmax != nullptr) {
            float run = g;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float v = __shfl_up_sync(0xffffffffu, run, o);
                if (lane >= o) run = fmaxf(run, v);
            }
            run = fmaxf(run, mx);
            mx = __shfl_sync(0xffffffffu, run, 31);
            gmax[t] = run;
        }
    }
}

__host__ __device__ constexpr int round16(int n) { return (n + 15) / 16 * 16; }

// grid (chunks, H)
template <int KIND>
__global__ void __launch_bounds__(G_THREADS, 2)
gm_chunk_state_kernel(const bf16* __restrict__ p, const bf16* __restrict__ w2, const float* __restrict__ bias, GmScratch sc,
                      const int* __restrict__ cu_q, GmArgs a) {
    extern __shared__ __align__(16) unsigned char smraw[];
    griddep_wait();
    int b, tile;
    const int flat = blockIdx.x, h = blockIdx.y;
    if (!find_query_tile(cu_q, a.B, GC, flat, b, tile)) return;
    const int t0 = cu_q[b] + tile * GC, nt = min(GC, cu_q[b + 1] - t0);
    const int dim = a.dim, vd = a.vd, dimP = round16(dim), vdP = round16(vd), rankP = round16(a.rank);
    const int LK = dimP + 8, LV = vdP + 8, LR = rankP + 8, LZ = dimP + 4;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    bf16* kh = reinterpret_cast<bf16*>(smraw);                 // [GC][LK]
    bf16* kl = kh + GC * LK;                                   // [GC][LK]
    bf16* vs = kl + GC * LK;                                   // [GC][LV]
    float* zb = reinterpret_cast<float*>(vs + GC * LV);        // GLA: [GC][LZ] the running sums; MLSTM: F, g
    float* seg = zb + (KIND == GLA ? GC * LZ : 2 * GC);        // GLA: [4][dimP]
    bf16* r1 = reinterpret_cast<bf16*>(seg + 4 * dimP);        // GLA: [GC][LR] the narrow rows
    bf16* r2 = r1 + GC * LR;                                   // GLA: [dimP][LR] W_2's rows of this head
    const bf16* prow = p + (size_t)t0 * a.ld;
    load_tile(vs, LV, prow + a.v_off + h * vd, a.ld, nt, vd, vdP);
    uint4 k_raw[4];                                            // the thread's first pieces of k, on their way from here on
    {
        const Pieces pc = pieces_of(tid, nt, dim, dimP);
#pragma unroll
        for (int u = 0; u < 4; u++) k_raw[u] = pc.in[u] ? *reinterpret_cast<const uint4*>(prow + (size_t)pc.t[u] * a.ld + a.k_off + h * dim + pc.c[u]) : make_uint4(0u, 0u, 0u, 0u);
    }
    if (KIND == GLA) {
        if (a.rank % 8 == 0 && a.a_off % 8 == 0) {             // (w2 is 16-byte aligned)
            const int ch = rankP / 8;
            for (int i = tid; i < (GC + dimP) * ch; i += G_THREADS) {
                const int r = i / ch, c = (i % ch) * 8;
                uint4 v = make_uint4(0u, 0u, 0u, 0u);
                if (r < GC) {
                    if (r < nt && c < a.rank) v = *reinterpret_cast<const uint4*>(prow + (size_t)r * a.ld + a.a_off + c);
                    *reinterpret_cast<uint4*>(r1 + r * LR + c) = v;
                } else {
                    if (r - GC < dim && c < a.rank) v = *reinterpret_cast<const uint4*>(w2 + (size_t)(h * dim + r - GC) * a.rank + c);
                    *reinterpret_cast<uint4*>(r2 + (r - GC) * LR + c) = v;
                }
            }
        } else
        for (int i = tid; i < (GC + dimP) * rankP; i += G_THREADS) {
            const int r = i / rankP, c = i % rankP;
            if (r < GC) r1[r * LR + c] = (r < nt && c < a.rank) ? prow[(size_t)r * a.ld + a.a_off + c] : __float2bfloat16_rn(0.f);
            else r2[(r - GC) * LR + c] = (r - GC < dim && c < a.rank) ? w2[(size_t)(h * dim + r - GC) * a.rank + c] : __float2bfloat16_rn(0.f);
        }
        __syncthreads();
        const uint32_t r1a = smem_u32(r1), r2a = smem_u32(r2);
        for (int item = warp; item < 4 * (dimP / 16); item += G_THREADS / 32) {
            const int m0 = (item & 3) * 16, n0 = (item >> 2) * 16;
            float c[2][4] = {};
            for (int k0 = 0; k0 < rankP; k0 += 16) {
                uint32_t af[4], bfr[4];
                ldmatrix_x4(af, addr_a(r1a, LR, m0, k0, lane));
                ldmatrix_x4(bfr, addr_b(r2a, LR, n0, k0, lane));
                mma_bf16(c[0], af, bfr[0], bfr[1]);
                mma_bf16(c[1], af, bfr[2], bfr[3]);
            }
#pragma unroll
            for (int j = 0; j < 2; j++)
#pragma unroll
                for (int e = 0; e < 4; e++)
                    zb[(m0 + (lane >> 2) + (e >> 1) * 8) * LZ + n0 + j * 8 + (lane & 3) * 2 + (e & 1)] = c[j][e];
        }
        __syncthreads();
        for (int i = tid; i < 4 * dim; i += G_THREADS) {       // running sums over 16 tokens at a time
            const int c = i % dim, s = i / dim;
            const float bc = bias[h * dim + c];
            float run = 0.f;
#pragma unroll 4
            for (int t = s * 16; t < s * 16 + 16; t++) {
                if (t < nt) run = fmaf(log2_sigmoid(zb[t * LZ + c] + bc), a.inv_tau, run);
                zb[t * LZ + c] = run;
            }
            seg[s * dimP + c] = run;
        }
        __syncthreads();
        for (int i = tid; i < GC * (dim / 4); i += G_THREADS) {        // the sums of the 16s before; out to memory
            const int t = i / (dim / 4), c = (i % (dim / 4)) * 4;
            float4 v = *reinterpret_cast<const float4*>(zb + t * LZ + c);
            for (int s = 0; s < t / 16; s++) {
                const float4 g = *reinterpret_cast<const float4*>(seg + s * dimP + c);
                v.x += g.x; v.y += g.y; v.z += g.z; v.w += g.w;
            }
            *reinterpret_cast<float4*>(zb + t * LZ + c) = v;
            if (t < nt) *reinterpret_cast<float4*>(sc.b + ((size_t)(t0 + t) * a.H + h) * dim + c) = v;
        }
    } else if (KIND == MLSTM) {
        mlstm_gates(p, bias, t0, nt, h, a, zb, zb + GC, nullptr);
    }
    __syncthreads();
    // k times its decay to the chunk's end, in two summands
    float G = -INFINITY;
    if (KIND == MLSTM) {
        for (int t = 0; t < GC; t++) G = fmaxf(G, zb[GC + t]);
        if (tid == 0) {
            sc.scal[((size_t)flat * a.H + h) * 2] = zb[nt - 1];
            sc.scal[((size_t)flat * a.H + h) * 2 + 1] = zb[nt - 1] + G;
        }
    }
    for (int i0 = tid; i0 < GC * (dimP / 8); i0 += 4 * G_THREADS) {
        const Pieces pc = pieces_of(i0, nt, dim, dimP);
        if (i0 != tid) {
#pragma unroll
            for (int u = 0; u < 4; u++) k_raw[u] = pc.in[u] ? *reinterpret_cast<const uint4*>(prow + (size_t)pc.t[u] * a.ld + a.k_off + h * dim + pc.c[u]) : make_uint4(0u, 0u, 0u, 0u);
        }
#pragma unroll
        for (int u = 0; u < 4; u++) {
            if (!pc.on[u]) continue;
            const int t = pc.t[u], c = pc.c[u];
            float kv[8];
            widen8(k_raw[u], kv);
            if (pc.in[u]) {
                if (KIND == GLA) {
                    float be[8], bt[8];
                    load8(zb + (nt - 1) * LZ + c, be);
                    load8(zb + t * LZ + c, bt);
#pragma unroll
                    for (int j = 0; j < 8; j++) kv[j] *= exp2f(be[j] - bt[j]);
                } else {
                    const float w = KIND == FIXED ? exp2f(bias[a.H + h] * (float)(nt - 1 - t)) : expf(zb[GC + t] - G);
#pragma unroll
                    for (int j = 0; j < 8; j++) kv[j] *= w;
                }
            }
            uint4 hi, lo;
            split8(kv, hi, lo);
            *reinterpret_cast<uint4*>(kh + t * LK + c) = hi;
            *reinterpret_cast<uint4*>(kl + t * LK + c) = lo;
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    const size_t fh = (size_t)flat * a.H + h;
    if (KIND == MLSTM) {
        for (int c = tid; c < dim; c += G_THREADS) {
            float s = 0.f;
            for (int t = 0; t < nt; t++) s += to_f32(kh[t * LK + c]) + to_f32(kl[t * LK + c]);
            sc.un[fh * dim + c] = s;
        }
    }
    // U = (decayed k)^T v: a warp takes 16 columns and every `ms`-th group of 16 rows
    float* U = sc.U + fh * dim * vd;
    const uint32_t kha = smem_u32(kh), kla = smem_u32(kl), va = smem_u32(vs);
    const int ncg = vdP / 16, ms = ncg >= 8 ? 1 : 8 / ncg;
    for (int item = warp; item < ncg * ms; item += G_THREADS / 32) {
        const int n0 = (item % ncg) * 16;
        uint32_t vf[4][4];
#pragma unroll
        for (int k = 0; k < 4; k++) ldmatrix_x4_trans(vf[k], addr_bt(va, LV, k * 16, n0, lane));
        for (int m0 = (item / ncg) * 16; m0 < dimP; m0 += ms * 16) {
            float c[2][4] = {};
#pragma unroll
            for (int k = 0; k < 4; k++) {
                uint32_t af[4];
                ldmatrix_x4_trans(af, addr_at(kha, LK, k * 16, m0, lane));
                mma_bf16(c[0], af, vf[k][0], vf[k][1]);
                mma_bf16(c[1], af, vf[k][2], vf[k][3]);
                ldmatrix_x4_trans(af, addr_at(kla, LK, k * 16, m0, lane));
                mma_bf16(c[0], af, vf[k][0], vf[k][1]);
                mma_bf16(c[1], af, vf[k][2], vf[k][3]);
            }
#pragma unroll
            for (int j = 0; j < 2; j++) {
                const int cc = n0 + j * 8 + (lane & 3) * 2;
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int r = m0 + (lane >> 2) + e * 8;
                    if (r < dim && cc < vd) *reinterpret_cast<float2*>(U + (size_t)r * vd + cc) = make_float2(c[j][2 * e], c[j][2 * e + 1]);
                }
            }
        }
    }
}

constexpr int SCAN_THREADS = 128;
constexpr int SCAN_AHEAD = 4;           // chunks whose U is in flight

// grid (groups of 4 * SCAN_THREADS entries of S, and behind them of n, H, B)
template <int KIND>
__global__ void __launch_bounds__(SCAN_THREADS)
gm_chunk_scan_kernel(GmState st, GmScratch sc, const float* __restrict__ bias, const int* __restrict__ cu_q, const int* __restrict__ slots, GmArgs a) {
    griddep_wait();
    const int h = blockIdx.y, b = blockIdx.z;
    const int slot = slots[b], q0 = cu_q[b], q1 = cu_q[b + 1];
    if (q1 <= q0) return;
    const int lane = threadIdx.x & 31;
    int base = 0;                                              // chunks of the sequences before this one
    for (int s = lane; s < b; s += 32) base += (cu_q[s + 1] - cu_q[s] + GC - 1) / GC;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) base += __shfl_xor_sync(0xffffffffu, base, o);
    const int nch = (q1 - q0 + GC - 1) / GC;
    const int nS = a.dim * a.vd / 4, nN = KIND == MLSTM ? a.dim / 4 : 0;
    const int e = blockIdx.x * SCAN_THREADS + threadIdx.x;
    if (e >= nS + nN) return;
    const bool is_n = e >= nS;
    const bool live = slot >= 0 && slot < a.n_slots;
    const size_t sh = (size_t)(live ? slot : 0) * a.H + h;
    const int row = is_n ? 0 : e * 4 / a.vd;
    float* stp = is_n ? st.n + sh * a.dim + (size_t)(e - nS) * 4 : st.S + sh * a.dim * a.vd + (size_t)e * 4;
    // chunk c of the sequence is chunk number base + nch - 1 - c of the step
    auto u_of = [&](int c) {
        const size_t fh = (size_t)(base + nch - 1 - c) * a.H + h;
        return reinterpret_cast<float4*>(is_n ? sc.un + fh * a.dim + (size_t)(e - nS) * 4 : sc.U + fh * a.dim * a.vd + (size_t)e * 4);
    };
    float4 S = live ? *reinterpret_cast<const float4*>(stp) : make_float4(0.f, 0.f, 0.f, 0.f);
    float m = KIND == MLSTM && live ? st.m[sh] : 0.f;
    const float lg = KIND == FIXED ? bias[a.H + h] : 0.f;
    float4 u[SCAN_AHEAD], un[SCAN_AHEAD];
    float2 d[SCAN_AHEAD], dn[SCAN_AHEAD];
    auto fetch = [&](int c0, float4 (&uu)[SCAN_AHEAD], float2 (&dd)[SCAN_AHEAD]) {
#pragma unroll
        for (int i = 0; i < SCAN_AHEAD; i++) {
            const int c = c0 + i;
            if (c >= nch) continue;
            uu[i] = *u_of(c);
            if (KIND == GLA) dd[i].x = sc.b[((size_t)(min(q0 + (c + 1) * GC, q1) - 1) * a.H + h) * a.dim + row];
            else if (KIND == FIXED) dd[i].x = lg * (float)(min(q0 + (c + 1) * GC, q1) - (q0 + c * GC));
            else dd[i] = *reinterpret_cast<const float2*>(sc.scal + ((size_t)(base + nch - 1 - c) * a.H + h) * 2);
        }
    };
    fetch(0, u, d);
    for (int c0 = 0; c0 < nch; c0 += SCAN_AHEAD) {
        fetch(c0 + SCAN_AHEAD, un, dn);
#pragma unroll
        for (int i = 0; i < SCAN_AHEAD; i++) {
            const int c = c0 + i;
            if (c >= nch) continue;
            *u_of(c) = S;                                      // the state before the chunk
            float keep, add = 1.f;
            if (KIND != MLSTM) {
                keep = exp2f(d[i].x);
            } else {
                if (e == 0) sc.m0[(size_t)(base + nch - 1 - c) * a.H + h] = m;
                const float m_new = fmaxf(m + d[i].x, d[i].y);
                keep = expf(m + d[i].x - m_new);
                add = expf(d[i].y - m_new);
                m = m_new;
            }
            S.x = fmaf(keep, S.x, add * u[i].x);
            S.y = fmaf(keep, S.y, add * u[i].y);
            S.z = fmaf(keep, S.z, add * u[i].z);
            S.w = fmaf(keep, S.w, add * u[i].w);
        }
#pragma unroll
        for (int i = 0; i < SCAN_AHEAD; i++) {
            u[i] = un[i];
            d[i] = dn[i];
        }
    }
    if (live) *reinterpret_cast<float4*>(stp) = S;
    // st.m is read by every thread of the head above; gm_chunk_out's first CTA of the sequence's last chunk writes it
}

// grid (chunks, H). NG: groups of 128 value columns.
template <int KIND, int NG>
__global__ void __launch_bounds__(G_THREADS, NG == 1 ? 2 : 1)
gm_chunk_out_kernel(const bf16* __restrict__ p, const float* __restrict__ bias, const float* __restrict__ w_norm, GmState st, GmScratch sc,
                    bf16* __restrict__ out, const int* __restrict__ cu_q, const int* __restrict__ slots, GmArgs a) {
    extern __shared__ __align__(16) unsigned char smraw[];
    __shared__ float Fs[GC], gs[GC], Ms[GC], den[GC], rsum[2][GC], ssq[8][GC];
    __shared__ int wide_s;
    griddep_wait();
    int b, tile;
    const int flat = blockIdx.x, h = blockIdx.y;
    if (!find_query_tile(cu_q, a.B, GC, flat, b, tile)) return;
    const int t0 = cu_q[b] + tile * GC, nt = min(GC, cu_q[b + 1] - t0);
    const int dim = a.dim, vd = a.vd, dimP = round16(dim), vdP = round16(vd);
    const int LK = dimP + 8, LV = vdP + 8;
    constexpr int LA = GC + 8, NQ = KIND == GLA ? 2 : 1;       // NQ: summands of q and k
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    bf16* qs = reinterpret_cast<bf16*>(smraw);                 // [NQ][GC][LK]
    bf16* vs = qs + NQ * GC * LK;                              // [GC][LV]
    float* rf = reinterpret_cast<float*>(vs + GC * LV);        // GLA: [dimP] factor of S's rows; MLSTM: n before the chunk
    bf16* ks = reinterpret_cast<bf16*>(rf + dimP);             // [NQ][GC][LK]; the scores lie there afterwards
    bf16* As = ks;                                             // [2][GC][LA]
    const bf16* prow = p + (size_t)t0 * a.ld;
    const size_t fh = (size_t)flat * a.H + h;
    float m0 = 0.f;
    const float lg = KIND == FIXED ? bias[a.H + h] : 0.f;      // binary logarithm of the head's decay
    uint4 q_raw[4], k_raw[4];
    float4 b_raw[4][2];
    auto fetch_qkb = [&](const Pieces& pc) {
#pragma unroll
        for (int u = 0; u < 4; u++) {
            q_raw[u] = k_raw[u] = make_uint4(0u, 0u, 0u, 0u);
            b_raw[u][0] = b_raw[u][1] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (pc.in[u]) {
                q_raw[u] = *reinterpret_cast<const uint4*>(prow + (size_t)pc.t[u] * a.ld + a.q_off + h * dim + pc.c[u]);
                k_raw[u] = *reinterpret_cast<const uint4*>(prow + (size_t)pc.t[u] * a.ld + a.k_off + h * dim + pc.c[u]);
                const float4* bp = reinterpret_cast<const float4*>(sc.b + ((size_t)(t0 + pc.t[u]) * a.H + h) * dim + pc.c[u]);
                b_raw[u][0] = bp[0];
                b_raw[u][1] = bp[1];
            }
        }
    };
    if (KIND == GLA) {
        fetch_qkb(pieces_of(tid, nt, dim, dimP));
        if (tid == 0) wide_s = 0;
        __syncthreads();
        const float* blast = sc.b + ((size_t)(t0 + nt - 1) * a.H + h) * dim;
        for (int c = tid; c < dimP; c += G_THREADS) {
            const float bl = c < dim ? blast[c] : 0.f;
            if (bl < -GLA_RANGE) wide_s = 1;
            rf[c] = 0.5f * bl;                                 // the channel's reference
        }
        __syncthreads();
        const bool wide = wide_s != 0;
        for (int i0 = tid; i0 < GC * (dimP / 8); i0 += 4 * G_THREADS) {
            const Pieces pc = pieces_of(i0, nt, dim, dimP);
            if (i0 != tid) fetch_qkb(pc);
#pragma unroll
            for (int u = 0; u < 4; u++) {
                if (!pc.on[u]) continue;
                const int t = pc.t[u], c = pc.c[u];
                float qv[8], kv[8], ref[8];
                widen8(q_raw[u], qv);
                widen8(k_raw[u], kv);
                const float bv[8] = {b_raw[u][0].x, b_raw[u][0].y, b_raw[u][0].z, b_raw[u][0].w, b_raw[u][1].x, b_raw[u][1].y, b_raw[u][1].z, b_raw[u][1].w};
                load8(rf + c, ref);
#pragma unroll
                for (int j = 0; j < 8; j++) {
                    const float x = wide ? bv[j] : bv[j] - ref[j];
                    qv[j] *= a.q_scale * exp2f(x);
                    if (!wide) kv[j] *= exp2f(-x);
                }
                uint4 hi, lo;
                split8(qv, hi, lo);
                *reinterpret_cast<uint4*>(qs + t * LK + c) = hi;
                *reinterpret_cast<uint4*>(qs + GC * LK + t * LK + c) = lo;
                if (!wide) {
                    split8(kv, hi, lo);
                    *reinterpret_cast<uint4*>(ks + t * LK + c) = hi;
                    *reinterpret_cast<uint4*>(ks + GC * LK + t * LK + c) = lo;
                }
            }
        }
        load_tile(vs, LV, prow + a.v_off + h * vd, a.ld, nt, vd, vdP);          // under the scores
    } else {
        load_tile(qs, LK, prow + a.q_off + h * dim, a.ld, nt, dim, dimP);
        load_tile(ks, LK, prow + a.k_off + h * dim, a.ld, nt, dim, dimP);
        load_tile(vs, LV, prow + a.v_off + h * vd, a.ld, nt, vd, vdP);
        if (KIND == MLSTM) {
            m0 = sc.m0[fh];
            mlstm_gates(p, bias, t0, nt, h, a, Fs, gs, Ms);
            for (int c = tid; c < dimP; c += G_THREADS) rf[c] = c < dim ? sc.un[fh * dim + c] : 0.f;
        }
        cp_async_wait<1>();                                    // q and k (the values land under the scores)
    }
    __syncthreads();
    const bool wide = KIND == GLA && wide_s != 0;
    if (KIND == MLSTM && tid < GC) Ms[tid] = fmaxf(Ms[tid], m0);       // (read by others behind the next barrier)
    if (KIND == GLA)                                                   // from here on the factor itself, for the state's rows
        for (int c = tid; c < dimP; c += G_THREADS) rf[c] = exp2f(rf[c]);
    // ---- scores: warp w takes tokens [16 (w & 3), +16) and keys [32 (w >> 2), +32)
    float s[4][4] = {};
    {
        const int m0r = (warp & 3) * 16, n0 = (warp >> 2) * 32;
        const bool none = n0 > m0r + 15;
        if (!none && !wide) {
            const uint32_t qa = smem_u32(qs), ka = smem_u32(ks);
            for (int k0 = 0; k0 < dimP; k0 += 16) {
                uint32_t af[NQ][4], bfr[NQ][2][4];
#pragma unroll
                for (int x = 0; x < NQ; x++) {
                    ldmatrix_x4(af[x], addr_a(qa + x * GC * LK * 2, LK, m0r, k0, lane));
#pragma unroll
                    for (int y = 0; y < 2; y++) ldmatrix_x4(bfr[x][y], addr_b(ka + x * GC * LK * 2, LK, n0 + y * 16, k0, lane));
                }
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    mma_bf16(s[j], af[0], bfr[0][j >> 1][(j & 1) * 2], bfr[0][j >> 1][(j & 1) * 2 + 1]);
                    if (NQ == 2) {
                        mma_bf16(s[j], af[NQ - 1], bfr[0][j >> 1][(j & 1) * 2], bfr[0][j >> 1][(j & 1) * 2 + 1]);
                        mma_bf16(s[j], af[0], bfr[NQ - 1][j >> 1][(j & 1) * 2], bfr[NQ - 1][j >> 1][(j & 1) * 2 + 1]);
                    }
                }
            }
        }
        __syncthreads();                                       // the keys have been read: the scores go over them
        if (!wide) {
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int t = m0r + g + e * 8;
                float sum = 0.f;
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const int key = n0 + j * 8 + t4 * 2;
                    float x = key <= t ? s[j][2 * e] : 0.f, y = key + 1 <= t ? s[j][2 * e + 1] : 0.f;
                    if (KIND == MLSTM) {                       // g_s <= M_t for s <= t; rows beyond the chunk are not stored
                        x = key <= t ? x * a.q_scale * expf(gs[key] - Ms[t]) : 0.f;
                        y = key + 1 <= t ? y * a.q_scale * expf(gs[key + 1] - Ms[t]) : 0.f;
                        sum += x + y;
                    } else if (KIND == FIXED) {
                        x = key <= t ? x * a.q_scale * exp2f(lg * (float)(t - key)) : 0.f;
                        y = key + 1 <= t ? y * a.q_scale * exp2f(lg * (float)(t - key - 1)) : 0.f;
                    }
                    float rx, ry;
                    *reinterpret_cast<uint32_t*>(As + t * LA + key) = hi_pack(x, y, rx, ry);
                    *reinterpret_cast<uint32_t*>(As + GC * LA + t * LA + key) = pack_bf16(rx, ry);
                }
                if (KIND == MLSTM) {
                    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
                    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
                    if (t4 == 0) rsum[warp >> 2][t] = sum;
                }
            }
        } else {
            // channel by channel, a warp a (token, key): every exponent is a sum of log decays between the two, so <= 0
            for (int i = warp; i < GC * GC; i += G_THREADS / 32) {
                const int t = i / GC, key = i % GC;
                float acc = 0.f;
                if (key <= t && t < nt)
                    for (int c = lane; c < dim; c += 32) {
                        const float qv = to_f32(prow[(size_t)t * a.ld + a.q_off + h * dim + c]);
                        const float kv = to_f32(prow[(size_t)key * a.ld + a.k_off + h * dim + c]);
                        acc = fmaf(qv * kv, exp2f(sc.b[((size_t)(t0 + t) * a.H + h) * dim + c] - sc.b[((size_t)(t0 + key) * a.H + h) * dim + c]), acc);
                    }
                acc = warp_sum(acc) * a.q_scale;
                if (lane == 0) {
                    const bf16 hi = __float2bfloat16_rn(acc);
                    As[t * LA + key] = hi;
                    As[GC * LA + t * LA + key] = __float2bfloat16_rn(acc - to_f32(hi));
                }
            }
        }
    }
    if (KIND == MLSTM) {
        // q . n of the state before the chunk, four threads a token
        const int t = tid >> 2;
        float nq = 0.f;
        for (int c = tid & 3; c < dim; c += 4) nq = fmaf(to_f32(qs[t * LK + c]), rf[c], nq);
        nq += __shfl_xor_sync(0xffffffffu, nq, 1);
        nq += __shfl_xor_sync(0xffffffffu, nq, 2);
        __syncthreads();
        if ((tid & 3) == 0) {
            const float n = rsum[0][t] + rsum[1][t] + nq * a.q_scale * expf(m0 - Ms[t]);
            den[t] = 1.0f / (fmaxf(fabsf(n), expf(-(Fs[t] + Ms[t]))) + MLSTM_FLOOR);
        }
        if (tid == 0) {                                        // the sequence's m behind its last chunk
            const int slot = slots[b];
            if (t0 + nt == cu_q[b + 1] && slot >= 0 && slot < a.n_slots) st.m[(size_t)slot * a.H + h] = Fs[nt - 1] + Ms[nt - 1];
        }
    }
    cp_async_wait<0>();                                        // the values
    __syncthreads();
    // ---- outputs: a warp takes 16 columns of every group of 128 and every `parts`-th group of 16 tokens
    const int ncg = min(8, vdP / 16);
    const int parts = NG == 1 ? min(4, 8 / ncg) : 1;
    const int cg = warp % ncg, part = warp / ncg;
    const bool on = part < parts;
    const float* S0 = sc.U + fh * dim * vd;
    const uint32_t qa = smem_u32(qs), Aa = smem_u32(As), va = smem_u32(vs);
    float acc[NG][4][2][4];
#pragma unroll
    for (int ng = 0; ng < NG; ng++)
#pragma unroll
        for (int mt = 0; mt < 4; mt++)
#pragma unroll
            for (int j = 0; j < 2; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[ng][mt][j][e] = 0.f;
    if (on) {
#pragma unroll
        for (int ng = 0; ng < NG; ng++) {
            const int n0 = ng * 128 + cg * 16;
            if (n0 >= vdP) continue;
            float x[2][4], xn[2][4], xm[2][4];                 // S's values of a step of 16 rows: rows 2 t4, +1, +8, +9; two steps ahead
            auto fetch = [&](int k0, float (&v)[2][4]) {
#pragma unroll
                for (int j = 0; j < 2; j++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int r = k0 + t4 * 2 + (e & 1) + (e >> 1) * 8, c = n0 + j * 8 + g;
                        v[j][e] = (r < dim && c < vd) ? S0[(size_t)r * vd + c] : 0.f;
                    }
            };
            fetch(0, x);
            fetch(16, xn);                                     // (rows beyond dim give zeros, without a load)
            for (int k0 = 0; k0 < dimP; k0 += 16) {
                fetch(k0 + 32, xm);
                uint32_t bh[2][2], bl[2][2];
#pragma unroll
                for (int j = 0; j < 2; j++)
#pragma unroll
                    for (int e = 0; e < 2; e++) {
                        float u0 = x[j][2 * e], u1 = x[j][2 * e + 1];
                        if (KIND == GLA && !wide) {
                            const int r = k0 + t4 * 2 + e * 8;
                            u0 *= rf[r];
                            u1 *= rf[r + 1];
                        }
                        float r0, r1;
                        bh[j][e] = hi_pack(u0, u1, r0, r1);
                        bl[j][e] = pack_bf16(r0, r1);
                    }
#pragma unroll
                for (int mt = 0; mt < 4; mt++) {
                    if (parts > 1 && mt % parts != part) continue;
                    uint32_t af[4];
                    ldmatrix_x4(af, addr_a(qa, LK, mt * 16, k0, lane));
#pragma unroll
                    for (int j = 0; j < 2; j++) {
                        mma_bf16(acc[ng][mt][j], af, bh[j][0], bh[j][1]);
                        mma_bf16(acc[ng][mt][j], af, bl[j][0], bl[j][1]);
                    }
                    if (NQ == 2) {
                        ldmatrix_x4(af, addr_a(qa + GC * LK * 2, LK, mt * 16, k0, lane));
#pragma unroll
                        for (int j = 0; j < 2; j++) mma_bf16(acc[ng][mt][j], af, bh[j][0], bh[j][1]);
                    }
                }
#pragma unroll
                for (int j = 0; j < 2; j++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        x[j][e] = xn[j][e];
                        xn[j][e] = xm[j][e];
                    }
            }
            if (KIND != GLA) {
#pragma unroll
                for (int mt = 0; mt < 4; mt++) {
                    const int ta = mt * 16 + g;
                    const float f0 = a.q_scale * (KIND == FIXED ? exp2f(lg * (float)(ta + 1)) : expf(m0 - Ms[ta]));
                    const float f1 = a.q_scale * (KIND == FIXED ? exp2f(lg * (float)(ta + 9)) : expf(m0 - Ms[ta + 8]));
#pragma unroll
                    for (int j = 0; j < 2; j++) {
                        acc[ng][mt][j][0] *= f0; acc[ng][mt][j][1] *= f0;
                        acc[ng][mt][j][2] *= f1; acc[ng][mt][j][3] *= f1;
                    }
                }
            }
#pragma unroll
            for (int k = 0; k < 4; k++) {
                uint32_t vf[4];
                ldmatrix_x4_trans(vf, addr_bt(va, LV, k * 16, n0, lane));
#pragma unroll
                for (int mt = 0; mt < 4; mt++) {
                    if (mt < k || (parts > 1 && mt % parts != part)) continue;
#pragma unroll
                    for (int x2 = 0; x2 < 2; x2++) {
                        uint32_t af[4];
                        ldmatrix_x4(af, addr_a(Aa + x2 * GC * LA * 2, LA, mt * 16, k * 16, lane));
                        mma_bf16(acc[ng][mt][0], af, vf[0], vf[1]);
                        mma_bf16(acc[ng][mt][1], af, vf[2], vf[3]);
                    }
                }
            }
        }
        // ---- the denominators, and the sums of squares of the rows
#pragma unroll
        for (int mt = 0; mt < 4; mt++) {
            if (parts > 1 && mt % parts != part) continue;
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int t = mt * 16 + g + e * 8;
                const float d = KIND == MLSTM ? den[t] : 1.0f;
                float q2 = 0.f;
#pragma unroll
                for (int ng = 0; ng < NG; ng++)
#pragma unroll
                    for (int j = 0; j < 2; j++) {
                        float& u0 = acc[ng][mt][j][2 * e];
                        float& u1 = acc[ng][mt][j][2 * e + 1];
                        u0 *= d;
                        u1 *= d;
                        q2 = fmaf(u0, u0, fmaf(u1, u1, q2));   // (columns beyond vd are zeros)
                    }
                q2 += __shfl_xor_sync(0xffffffffu, q2, 1);
                q2 += __shfl_xor_sync(0xffffffffu, q2, 2);
                if (t4 == 0) ssq[cg][t] = q2;
            }
        }
    }
    __syncthreads();
    if (!on) return;
#pragma unroll
    for (int mt = 0; mt < 4; mt++) {
        if (parts > 1 && mt % parts != part) continue;
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int t = mt * 16 + g + e * 8;
            if (t >= nt) continue;
            float q2 = 0.f;                                    // (in the order of the columns)
            for (int w = 0; w < ncg; w++) q2 += ssq[w][t];
            const float r = 1.0f / sqrtf(q2 / (float)vd + a.eps);
#pragma unroll
            for (int ng = 0; ng < NG; ng++)
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    const int c = ng * 128 + cg * 16 + j * 8 + t4 * 2;
                    if (c >= vd) continue;
                    const __nv_bfloat162 z = *reinterpret_cast<const __nv_bfloat162*>(prow + (size_t)t * a.ld + a.g_off + h * vd + c);
                    const float2 w = *reinterpret_cast<const float2*>(w_norm + h * vd + c);
                    const float y0 = acc[ng][mt][j][2 * e] * r * w.x * gate_act<KIND>(__bfloat162float(z.x));
                    const float y1 = acc[ng][mt][j][2 * e + 1] * r * w.y * gate_act<KIND>(__bfloat162float(z.y));
                    *reinterpret_cast<uint32_t*>(out + (size_t)(t0 + t) * a.ldo + a.o_off + h * vd + c) = pack_bf16(y0, y1);
                }
        }
    }
}

template <typename T, int KIND>
int launch_token(const void* p, const void* w2, const float* bias, const float* w_norm, const GmState& st, void* out, const int* cu_q,
                 const int* slots, const GmArgs& a, int max_q_len, cudaStream_t stream) {
    const int vec = a.vd % 4 == 0 ? 4 : 1, cols = a.vd / vec;
    int nt = 128;
    while (nt < 512 && (nt < cols || (long long)a.dim * a.vd > (long long)nt * vec * TOK_BATCH)) nt <<= 1;
    MYNAH_REQUIRE(cols <= nt, "gated_memory: value heads of %d exceed what the token form lays across a block", a.vd);
    const int groups = nt / cols;
    const size_t base = (size_t)(3 * a.dim + 2 * a.vd + a.rank + 32 + 4 + groups * a.vd + a.dim + 4) * sizeof(float);
    const size_t full = base + (size_t)a.dim * a.vd * sizeof(float);
    const int in_smem = max_q_len > 1 && full <= 200 * 1024;
    const size_t smem = in_smem ? full : base;
    MYNAH_REQUIRE(smem <= 220 * 1024, "gated_memory: heads of %d x %d do not fit the token form", a.dim, a.vd);
    auto go = [&](auto kern) {
        if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
            return mynah_fail("gated_memory: %zu bytes of shared memory are not to be had", smem);
        mynah_launch(kern, dim3(a.H, a.B), dim3(nt), smem, stream, (const T*)p, (const T*)w2, bias, w_norm, st, (T*)out, cu_q, slots, a, in_smem);
        return mynah_check_launch("gated_memory (tokens)");
    };
    return vec == 4 ? go(gm_token_kernel<T, KIND, 4>) : go(gm_token_kernel<T, KIND, 1>);
}

template <int KIND>
int launch_chunks(const void* p, const void* w2, const float* bias, const float* w_norm, const GmState& st, const GmScratch& sc, void* out,
                  const int* cu_q, const int* slots, const GmArgs& a, int rows, cudaStream_t stream) {
    const int dimP = round16(a.dim), vdP = round16(a.vd), rankP = round16(a.rank);
    const int chunks = rows / GC + a.B;
    size_t smem = (size_t)(2 * GC * (dimP + 8) + GC * (vdP + 8)) * sizeof(bf16);
    if (KIND == GLA) smem += (size_t)(GC * (dimP + 4) + 4 * dimP) * sizeof(float) + (size_t)(GC + dimP) * (rankP + 8) * sizeof(bf16);
    else smem += (size_t)(2 * GC + 4 * dimP) * sizeof(float);
    MYNAH_REQUIRE(smem <= 220 * 1024, "gated_memory: heads of %d x %d with a narrow size of %d do not fit the chunk form", a.dim, a.vd, a.rank);
    auto k1 = gm_chunk_state_kernel<KIND>;
    if (smem > 48 * 1024 && cudaFuncSetAttribute(k1, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
        return mynah_fail("gated_memory: %zu bytes of shared memory are not to be had", smem);
    mynah_launch(k1, dim3(chunks, a.H), dim3(G_THREADS), smem, stream, (const bf16*)p, (const bf16*)w2, bias, sc, cu_q, a);
    if (mynah_check_launch("gated_memory (chunk states)") != 0) return -1;
    const int entries = a.dim * a.vd / 4 + (KIND == MLSTM ? a.dim / 4 : 0);
    mynah_launch(gm_chunk_scan_kernel<KIND>, dim3(ceil_div(entries, SCAN_THREADS), a.H, a.B), dim3(SCAN_THREADS), 0, stream, st, sc, bias, cu_q, slots, a);
    if (mynah_check_launch("gated_memory (chunk scan)") != 0) return -1;
    constexpr int NQ = KIND == GLA ? 2 : 1;
    const size_t keys = (size_t)NQ * GC * (dimP + 8), scores = (size_t)2 * GC * (GC + 8);
    const size_t smem_o = ((size_t)NQ * GC * (dimP + 8) + (size_t)GC * (vdP + 8) + (keys > scores ? keys : scores)) * sizeof(bf16) + (size_t)dimP * sizeof(float);
    MYNAH_REQUIRE(smem_o <= 220 * 1024, "gated_memory: heads of %d x %d do not fit the chunk form", a.dim, a.vd);
    auto go = [&](auto kern) {
        if (smem_o > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_o) != cudaSuccess)
            return mynah_fail("gated_memory: %zu bytes of shared memory are not to be had", smem_o);
        mynah_launch(kern, dim3(chunks, a.H), dim3(G_THREADS), smem_o, stream, (const bf16*)p, bias, w_norm, st, sc, (bf16*)out, cu_q, slots, a);
        return mynah_check_launch("gated_memory (chunk outputs)");
    };
    return vdP <= 128 ? go(gm_chunk_out_kernel<KIND, 1>) : go(gm_chunk_out_kernel<KIND, 2>);
}

}  // namespace

// 0: every step walks token by token; otherwise bfloat16 prompt steps whose longest piece has at least this many tokens go
// chunk by chunk.
static int g_gm_chunk_min = 16;
MYNAH_API int mynah_gated_memory_chunk_min(int n) {
    const int before = g_gm_chunk_min;
    g_gm_chunk_min = n;
    return before;
}

static bool gm_chunked(int dtype, int dim, int vd, int rank, int max_q_len) {
    return dtype == MYNAH_BF16 && g_gm_chunk_min > 0 && max_q_len > 1 && max_q_len >= g_gm_chunk_min && dim % 8 == 0 && vd % 8 == 0 &&
           dim <= 256 && vd <= 256 && rank <= 64;
}

// Floats of scratch that mynah_gated_memory wants for a step of `rows` rows in B sequences (0: it walks token by token).
// kind 0: GLA, 1: MLSTM, 2: FIXED.
MYNAH_API long long mynah_gated_memory_scratch_floats(int kind, int dtype, int rows, int B, int H, int dim, int vd, int rank, int max_q_len) {
    if (!gm_chunked(dtype, dim, vd, rank, max_q_len)) return 0;
    const long long fh = (long long)(rows / GC + B) * H;
    if (kind == FIXED) return fh * dim * vd;
    return kind == GLA ? fh * dim * vd + (long long)rows * H * dim : fh * ((long long)dim * vd + dim + 4);
}

// p: [rows][ld] rows whose columns hold, from q_off / k_off / v_off / g_off on, every head's q and k (dim values each), v and
// gate (vd each); kind 0 (GLA): the narrow row of `rank` values at a_off, w2 [H * dim][rank] in dtype and bias fp32 [H * dim];
// kind 1 (MLSTM): the heads' input gates at a_off and forget gates at b_off, bias fp32 [2 H] (input, then forget);
// kind 2 (FIXED): bias fp32 [2 H], the heads' decays (not negative), then their binary logarithms (a finite number below -1e4
// for a decay of zero).
// w_norm: fp32 [H * vd]. State fp32: S [n_slots + 1][H][dim][vd]; kind 1 also n [...][dim] and m [...]. out: [rows][ldo] in
// dtype. max_q_len: the most tokens a sequence brings. scratch: mynah_gated_memory_scratch_floats(...) floats, 16-byte aligned,
// or null (token by token).
MYNAH_API int mynah_gated_memory(int kind, const void* p, int ld, int q_off, int k_off, int v_off, int g_off, int a_off, int b_off, int dtype,
                                 const void* w2, int rank, const float* bias, const float* w_norm, float q_scale, float inv_tau, float cap,
                                 float eps, float* S, float* n, float* m, int n_slots, void* out, int ldo, int o_off, const int* cu_q,
                                 const int* slots, int B, int rows, int H, int dim, int vd, int max_q_len, float* scratch,
                                 cudaStream_t stream) {
    if (B == 0 || rows == 0) return 0;
    MYNAH_REQUIRE(kind == GLA || kind == MLSTM || kind == FIXED, "gated_memory: kind %d is none of 0, 1, 2", kind);
    MYNAH_REQUIRE(B > 0 && rows > 0 && H > 0 && dim > 0 && vd > 0 && H <= 65535 && B <= 65535, "gated_memory: bad sizes");
    MYNAH_REQUIRE(bias != nullptr && (kind == FIXED || (kind == GLA ? rank > 0 && w2 != nullptr : n != nullptr && m != nullptr && cap > 0.f)), "gated_memory: what the kind needs is missing");
    MYNAH_REQUIRE(dtype == MYNAH_F32 || dtype == MYNAH_BF16, "gated_memory: unsupported dtype %d", dtype);
    const GmArgs a{B, H, dim, vd, ld, ldo, o_off, q_off, k_off, v_off, g_off, a_off, b_off, kind == GLA ? rank : 0, n_slots, q_scale, inv_tau, cap, eps};
    const GmState st{S, n, m};
    const bool aligned = ld % 8 == 0 && ldo % 2 == 0 && o_off % 2 == 0 && q_off % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0 && g_off % 2 == 0 &&
                         (((uintptr_t)p | (uintptr_t)S | (uintptr_t)scratch) & 15) == 0 && (((uintptr_t)out & 3) | ((uintptr_t)w_norm & 7)) == 0;
    if (scratch != nullptr && aligned && gm_chunked(dtype, dim, vd, a.rank, max_q_len)) {
        const size_t fh = (size_t)(rows / GC + B) * H;
        GmScratch sc{};
        sc.U = scratch;
        if (kind == GLA) {
            sc.b = scratch + fh * dim * vd;
            return launch_chunks<GLA>(p, w2, bias, w_norm, st, sc, out, cu_q, slots, a, rows, stream);
        }
        if (kind == FIXED) return launch_chunks<FIXED>(p, w2, bias, w_norm, st, sc, out, cu_q, slots, a, rows, stream);
        sc.un = scratch + fh * dim * vd;
        sc.scal = sc.un + fh * dim;
        sc.m0 = sc.scal + 2 * fh;
        return launch_chunks<MLSTM>(p, w2, bias, w_norm, st, sc, out, cu_q, slots, a, rows, stream);
    }
    MYNAH_REQUIRE(kind != GLA || dtype == MYNAH_F32 || ((uintptr_t)w2 & 15) == 0, "gated_memory: the narrow matrix is not aligned");
    if (kind == FIXED)
        return dtype == MYNAH_F32 ? launch_token<float, FIXED>(p, w2, bias, w_norm, st, out, cu_q, slots, a, max_q_len, stream)
                                  : launch_token<bf16, FIXED>(p, w2, bias, w_norm, st, out, cu_q, slots, a, max_q_len, stream);
    if (dtype == MYNAH_F32)
        return kind == GLA ? launch_token<float, GLA>(p, w2, bias, w_norm, st, out, cu_q, slots, a, max_q_len, stream)
                           : launch_token<float, MLSTM>(p, w2, bias, w_norm, st, out, cu_q, slots, a, max_q_len, stream);
    return kind == GLA ? launch_token<bf16, GLA>(p, w2, bias, w_norm, st, out, cu_q, slots, a, max_q_len, stream)
                       : launch_token<bf16, MLSTM>(p, w2, bias, w_norm, st, out, cu_q, slots, a, max_q_len, stream);
}
