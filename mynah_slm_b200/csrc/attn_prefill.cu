// Causal grouped-query attention of a ragged batch over the paged cache:
// every query of the step reads the keys of its own sequence at positions
// <= its own (and > its own - window, when the layer has a window), wherever
// they were written: in this step or in earlier ones.
//
// This is the general kernel: any head_dim up to 256, any number of heads and
// groups, both precisions, any mix of query lengths (one token included). It
// is the only attention of the 32-bit path's prompts, and the fallback of the
// bf16 path for head sizes the tensor-core kernel does not take.
//
// Formulas: score = dot(q, k) * (1/sqrtf(head_dim)), scale after the dot;
// softmax with the maximum subtracted; out = sum_t p_t v_t; query head h
// reads kv head h / (H/KV)  (mynah-slm src/kernels.c:228-250, :207-220).
// Scores, softmax and the output sum are fp32. Keys are taken 32 at a time at
// positions that are multiples of 32, so a query's sum runs in the same
// order whatever else is in the batch.
#include "layout.cuh"

namespace {

constexpr int QT = 16;          // queries per CTA
constexpr int KT = 32;          // keys per tile (one per lane)
constexpr int WARPS = 4;
constexpr int QPW = QT / WARPS; // queries per warp
constexpr int MAXC = 8;         // head_dim <= 32 * MAXC

struct PrefillArgs {
    int B, H, KV, HD, ldq, ldo;
    int window;                 // 0: all keys
    float scale;
    int VD;                     // width of a value head (HD unless the mixer's values are narrower or wider)
    int chunk;                  // 0: none; C: a query at position p sees keys from floor(p / C) * C on
    float softcap;              // 0: none; c: score <- c * tanh(score / c), after the scale
    int keep_first;             // with a window: keys at positions below it stay visible whatever their distance
    int vdiv;                   // kv head g reads value head g / vdiv (1 unless several key heads share one value head)
    int null_key;               // 1: the softmax has one more term, of score 0 and without a value
    float out_scale;            // factor on the output rows
    int vdo;                    // columns of a head in the output rows (<= VD: padding columns of the values are left out)
    const float* sink;          // null, or that term's score a query head (neither scaled nor capped)
};

template <typename TA, typename TC>
__global__ void __launch_bounds__(WARPS * 32)
attn_prefill_generic_kernel(const TA* __restrict__ q, TA* __restrict__ out,
                            const TC* __restrict__ k_cache, const TC* __restrict__ v_cache,
                            const int* __restrict__ cu_q, const int* __restrict__ kv_len,
                            PageTable pt, PrefillArgs a, int* __restrict__ status) {
    extern __shared__ float smem[];
    const int HD = a.HD, VD = a.VD, KS = HD + 1;      // padded key rows: lanes read distinct banks
    float* Ks = smem;                                  // [KT][HD+1]
    float* Vs = Ks + KT * KS;                          // [KT][VD]
    float* Qs = Vs + KT * VD;                          // [QT][HD]

    int b, tile;
    if (!find_query_tile(cu_q, a.B, QT, blockIdx.x, b, tile)) return;   // blockIdx.x numbers the step's query tiles
    const int h = blockIdx.y;
    const int q0 = cu_q[b], q_len = cu_q[b + 1] - q0;
    const int tile0 = tile * QT;
    const int n_kv = kv_len[b];
    const int past = n_kv - q_len;                     // position of the sequence's first query
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kvh = h / (a.H / a.KV);
    const int nq = min(QT, q_len - tile0);

    for (int i = threadIdx.x; i < QT * HD; i += blockDim.x) {
        const int qi = i / HD, d = i % HD;
        Qs[i] = qi < nq ? to_f32(q[(size_t)(q0 + tile0 + qi) * a.ldq + (size_t)h * HD + d]) : 0.f;
    }

    float m[QPW], l[QPW], acc[QPW][MAXC];
#pragma unroll
    for (int i = 0; i < QPW; i++) {
        m[i] = -INFINITY;
        l[i] = 0.f;
#pragma unroll
        for (int c = 0; c < MAXC; c++) acc[i][c] = 0.f;
    }

    const int p_first = past + tile0, p_last = past + tile0 + nq - 1;
    int k_lo = 0;
    if (a.window > 0) k_lo = max(0, p_first - a.window + 1);
    if (a.chunk > 0) k_lo = max(k_lo, (p_first / a.chunk) * a.chunk);
    k_lo = (k_lo / KT) * KT;
    // kept first tokens: the tiles below `first_end` are walked too, the ones between them and the window skipped
    const int first_end = (a.window > 0 && a.keep_first > 0) ? a.keep_first : 0;
    const int KVV = a.KV / a.vdiv, vh = kvh / a.vdiv;

    for (int kt = first_end > 0 ? 0 : k_lo; kt <= p_last; kt += KT) {
        if (kt >= first_end && kt < k_lo) {            // uniform over the CTA
            kt = k_lo - KT;
            continue;
        }
        __syncthreads();                               // previous tile consumed; Qs written (first pass)
        const int page = page_of(pt, b, kt);
        if (page < 0) {
            if (threadIdx.x == 0) atomicOr(status, MYNAH_ST_PAGE_RANGE);
            return;                                    // uniform over the CTA
        }
        const size_t base = (((size_t)page * a.KV + kvh) * PAGE_TOKENS + kt % PAGE_TOKENS) * HD;
        const size_t vbase = (((size_t)page * KVV + vh) * PAGE_TOKENS + kt % PAGE_TOKENS) * VD;
        const int n_keys = min(KT, n_kv - kt);         // rows past the sequence's end are not read
        for (int i = threadIdx.x; i < KT * HD; i += blockDim.x) {
            const int j = i / HD, d = i % HD;
            Ks[j * KS + d] = j < n_keys ? to_f32(k_cache[base + i]) : 0.f;
        }
        for (int i = threadIdx.x; i < KT * VD; i += blockDim.x)
            Vs[i] = i / VD < n_keys ? to_f32(v_cache[vbase + i]) : 0.f;
        __syncthreads();

#pragma unroll
        for (int i = 0; i < QPW; i++) {
            const int qi = warp * QPW + i;
            if (qi >= nq) continue;                    // uniform over the warp
            const int p = past + tile0 + qi;
            const int key = kt + lane;
            const float* qrow = Qs + qi * HD;
            const float* krow = Ks + lane * KS;
            float dot = 0.f;
            for (int d = 0; d < HD; d++) dot = fmaf(qrow[d], krow[d], dot);
            bool vis = key <= p && key < n_kv;
            if (a.window > 0) vis = vis && (key > p - a.window || key < a.keep_first);
            if (a.chunk > 0) vis = vis && key >= (p / a.chunk) * a.chunk;
            float sc = dot * a.scale;
            if (a.softcap > 0.f) sc = a.softcap * tanhf(sc / a.softcap);
            const float s = vis ? sc : -INFINITY;
            const float m_new = fmaxf(m[i], warp_max(s));
            if (m_new == -INFINITY) continue;          // no visible key yet (uniform)
            const float alpha = expf(m[i] - m_new);    // exp(-inf) = 0 on the first tile
            const float pj = expf(s - m_new);
            l[i] = l[i] * alpha + warp_sum(pj);
            m[i] = m_new;
#pragma unroll
            for (int c = 0; c < MAXC; c++) acc[i][c] *= alpha;
            for (int j = 0; j < KT; j++) {
                const float pb = __shfl_sync(0xffffffffu, pj, j);
#pragma unroll
                for (int c = 0; c < MAXC; c++) {
                    const int d = lane + 32 * c;
                    if (d < VD) acc[i][c] = fmaf(pb, Vs[j * VD + d], acc[i][c]);
                }
            }
        }
    }

#pragma unroll
    for (int i = 0; i < QPW; i++) {
        const int qi = warp * QPW + i;
        if (qi >= nq) continue;
        // the term without a key counts exp(0 - m), or exp(sink - m); where that overflows, the keys' share of the softmax is zero
        float ls = l[i];
        if (a.sink != nullptr && ls > 0.f) ls += expf(a.sink[h] - m[i]);
        else if (a.null_key && ls > 0.f) ls += expf(-m[i]);
        const float inv = ls > 0.f ? a.out_scale / ls : 0.f;
        TA* o = out + (size_t)(q0 + tile0 + qi) * a.ldo + (size_t)h * a.vdo;
#pragma unroll
        for (int c = 0; c < MAXC; c++) {
            const int d = lane + 32 * c;
            if (d < a.vdo) o[d] = from_f32<TA>(acc[i][c] * inv);
        }
    }
}

}  // namespace

// The general form: value heads of their own width VD (out has head h at columns [h*VD, (h+1)*VD)), a score
// scale given by the caller (0: 1/sqrt(HD)), and a chunk mask (0: none) beside the window.
MYNAH_API int mynah_attn_prefill_generic_ex(
    const void* q, void* out, int dtype, int n_tokens, int B, int max_q_len, int H, int KV, int HD, int VD, int ldq, int ldo,
    const void* k_cache, const void* v_cache, const int* cu_q, const int* kv_len,
    const int* page_indptr, const int* page_ids, const int* page_base, int n_pages,
    int window, int chunk, float scale, int* status, cudaStream_t stream);

// The same with capped scores (softcap c > 0: score <- c tanh(score / c)), first tokens that a window keeps
// (keep_first), several key heads on one value head (the value cache has KV / vdiv heads), one more softmax term of score
// 0 that has no value (null_key) or of a score of its own for every query head (sink, fp32 [H]; neither scaled nor capped), a
// factor on the output (out_scale) and output heads of `vdo` columns (0: VD).
MYNAH_API int mynah_attn_prefill_generic_capped(
    const void* q, void* out, int dtype, int n_tokens, int B, int max_q_len, int H, int KV, int HD, int VD, int ldq, int ldo,
    const void* k_cache, const void* v_cache, const int* cu_q, const int* kv_len,
    const int* page_indptr, const int* page_ids, const int* page_base, int n_pages,
    int window, int chunk, float scale, float softcap, int keep_first, int vdiv, int null_key, const float* sink, float out_scale, int vdo,
    int* status, cudaStream_t stream);

// q: [T, ldq] with head h at columns [h*HD, (h+1)*HD); out: [T, ldo] likewise.
MYNAH_API int mynah_attn_prefill_generic(
    const void* q, void* out, int dtype, int n_tokens, int B, int max_q_len, int H, int KV, int HD, int ldq, int ldo,
    const void* k_cache, const void* v_cache, const int* cu_q, const int* kv_len,
    const int* page_indptr, const int* page_ids, const int* page_base, int n_pages,
    int window, int* status, cudaStream_t stream) {
    return mynah_attn_prefill_generic_ex(q, out, dtype, n_tokens, B, max_q_len, H, KV, HD, HD, ldq, ldo, k_cache, v_cache,
                                         cu_q, kv_len, page_indptr, page_ids, page_base, n_pages, window, 0, 0.f, status,
                                         stream);
}

MYNAH_API int mynah_attn_prefill_generic_ex(
    const void* q, void* out, int dtype, int n_tokens, int B, int max_q_len, int H, int KV, int HD, int VD, int ldq, int ldo,
    const void* k_cache, const void* v_cache, const int* cu_q, const int* kv_len,
    const int* page_indptr, const int* page_ids, const int* page_base, int n_pages,
    int window, int chunk, float scale, int* status, cudaStream_t stream) {
    return mynah_attn_prefill_generic_capped(q, out, dtype, n_tokens, B, max_q_len, H, KV, HD, VD, ldq, ldo, k_cache, v_cache,
                                             cu_q, kv_len, page_indptr, page_ids, page_base, n_pages, window, chunk, scale,
                                             0.f, 0, 1, 0, nullptr, 1.0f, VD, status, stream);
}

MYNAH_API int mynah_attn_prefill_generic_capped(
    const void* q, void* out, int dtype, int n_tokens, int B, int max_q_len, int H, int KV, int HD, int VD, int ldq, int ldo,
    const void* k_cache, const void* v_cache, const int* cu_q, const int* kv_len,
    const int* page_indptr, const int* page_ids, const int* page_base, int n_pages,
    int window, int chunk, float scale, float softcap, int keep_first, int vdiv, int null_key, const float* sink, float out_scale, int vdo,
    int* status, cudaStream_t stream) {
    if (B == 0 || max_q_len == 0) return 0;
    MYNAH_REQUIRE(softcap >= 0.f && keep_first >= 0 && vdiv >= 1 && KV % vdiv == 0, "attn_prefill: bad cap, kept tokens or value sharing");
    MYNAH_REQUIRE(keep_first == 0 || chunk == 0, "attn_prefill: kept first tokens and a chunk mask do not go together");
    MYNAH_REQUIRE(B > 0 && H > 0 && KV > 0 && HD > 0 && H % KV == 0, "attn_prefill: bad sizes B=%d H=%d KV=%d HD=%d", B, H, KV, HD);
    MYNAH_REQUIRE(HD <= 32 * MAXC, "attn_prefill: head_dim %d exceeds %d", HD, 32 * MAXC);
    MYNAH_REQUIRE(VD > 0 && VD <= 32 * MAXC, "attn_prefill: value head of %d lies outside 1..%d", VD, 32 * MAXC);
    MYNAH_REQUIRE(vdo >= 0 && vdo <= VD, "attn_prefill: %d output columns a head exceed the value head of %d", vdo, VD);
    MYNAH_REQUIRE(chunk >= 0, "attn_prefill: negative chunk");
    MYNAH_REQUIRE(H <= 65535, "attn_prefill: H=%d exceeds one launch", H);
    MYNAH_REQUIRE(window >= 0, "attn_prefill: negative window");
    const PrefillArgs a{B, H, KV, HD, ldq, ldo, window, scale != 0.f ? scale : 1.0f / sqrtf((float)HD), VD, chunk, softcap, keep_first, vdiv,
                        null_key, out_scale, vdo > 0 ? vdo : VD, sink};
    const PageTable pt{page_indptr, page_ids, page_base, n_pages};
    const size_t smem = sizeof(float) * ((size_t)KT * (HD + 1) + (size_t)KT * VD + (size_t)QT * HD);
    (void)max_q_len;
    MYNAH_REQUIRE(n_tokens >= 0, "attn_prefill: negative row count");
    const dim3 grid(ceil_div(n_tokens, QT) + B, H, 1);               // the most query tiles that n_tokens rows in B sequences make
    cudaError_t e = cudaSuccess;
    if (dtype == MYNAH_F32) {
        auto kern = attn_prefill_generic_kernel<float, float>;
        if (smem > 48 * 1024) e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return mynah_fail("attn_prefill: %s", cudaGetErrorString(e));
        kern<<<grid, WARPS * 32, smem, stream>>>((const float*)q, (float*)out, (const float*)k_cache,
                                                 (const float*)v_cache, cu_q, kv_len, pt, a, status);
    } else if (dtype == MYNAH_BF16) {
        auto kern = attn_prefill_generic_kernel<bf16, bf16>;
        if (smem > 48 * 1024) e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return mynah_fail("attn_prefill: %s", cudaGetErrorString(e));
        kern<<<grid, WARPS * 32, smem, stream>>>((const bf16*)q, (bf16*)out, (const bf16*)k_cache,
                                                 (const bf16*)v_cache, cu_q, kv_len, pt, a, status);
    } else {
        return mynah_fail("attn_prefill: unsupported dtype %d", dtype);
    }
    return mynah_check_launch("attn_prefill_generic");
}
