// Helpers shared by the tensor-core attention kernels (decode and prefill):
// cp.async staging, ldmatrix, the bf16 m16n8k16 product, and the swizzled layout
// of a [64][head_dim] tile in shared memory.
#pragma once
#include "common.cuh"

__device__ __forceinline__ void dec_cp_async16(void* smem, const void* gmem) {
    if (!ZLM_CHK(gmem, 16)) return;
    const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(s), "l"(gmem));
}
__device__ __forceinline__ void dec_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void dec_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }

__device__ __forceinline__ void dec_ldsm4(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const void* p) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(s));
}
__device__ __forceinline__ void dec_ldsm4t(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const void* p) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(s));
}
__device__ __forceinline__ void dec_mma(float* c, const unsigned* a, unsigned b0, unsigned b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *(unsigned*)&v;
}

// What a mixer may ask of the attention kernels beyond the scale and the window.
//   chunk    > 0: a query sees only the keys of its own chunk of that many positions, counted from position 0
//   softcap  > 0: scores become softcap * tanh(score * scale / softcap)
//   sinks    one number per query head whose exponential joins the softmax's denominator without a value
//            (null with the flag `sink` set: the number is 0)
//   v_share  that many neighbouring key heads read one value head: a page is [nkv key heads | nkv / v_share value
//            heads] of [ZLM_PAGE][hd] each (1: the ordinary [K | V] of nkv heads each)
//   keep     > 0 (with a window): the sequence's first `keep` positions stay visible beside the window
//   bias     numbers added to the scores after scale and cap, by distance: bias_n of them a head, query i reads the
//            min(i - j, bias_n - 1)-th for key j.  A head's row of the table is [ATTN_BIAS_LEAD | bias_n | ATTN_BIAS_TAIL]
//            floats: what comes before the first number is never used, what follows repeats the last one, so that a tile
//            with a distance below bias_n - 1 in it reads the table at pos - key for all its keys, seen or not
struct AttnOpts {
    int chunk;
    float softcap;
    const float* sinks;
    int v_share;
    int keep;
    const float* bias;
    int bias_n;
};
static inline AttnOpts attn_no_opts() { return AttnOpts{0, 0.f, nullptr, 1, 0, nullptr, 0}; }
// what the entry points ask of the options they are given
#define ZLM_REQUIRE_ATTN_OPTS(what)                                                                                   \
    ZLM_REQUIRE(chunk >= 0 && softcap >= 0.f && v_share >= 1 && nkv % v_share == 0,                                   \
                what ": chunk=%d softcap=%g v_share=%d", chunk, (double)softcap, v_share);                            \
    ZLM_REQUIRE(keep >= 0 && (keep == 0 || (window > 0 && chunk == 0)), what ": %d first keys beside a window of %d", keep, window); \
    ZLM_REQUIRE(!bias || bias_n > 0, what ": a distance bias of %d entries", bias_n)
#define ATTN_LOG2E 1.4426950408889634f

// the first key that the query at `pos` reads
__device__ __forceinline__ int attn_first_key(int pos, int window, int chunk) {
    int lo = (window != 0 && pos + 1 > window) ? pos + 1 - window : 0;
    if (chunk > 0) lo = max(lo, pos - pos % chunk);
    return lo;
}

// The pages a tile of queries walks: the pages of the first kept keys, then those from the tile's first key on.
//   n        how many
//   page(w)  the w-th one's logical page; beyond the last one, pages beyond every query's position
struct AttnWalk {
    int kept, lo, n;
    __device__ __forceinline__ AttnWalk(int page_lo, int page_hi, int keep) {
        kept = keep > 0 ? min((keep + ZLM_PAGE - 1) / ZLM_PAGE, page_hi) : 0;
        lo = keep > 0 ? max(page_lo, kept) : page_lo;
        n = kept + page_hi - lo;
    }
    __device__ __forceinline__ int page(int w) const { return w < kept ? w : lo + (w - kept); }
};

// whether the query at `pos` whose window starts at `lo` reads the key
__device__ __forceinline__ bool attn_sees(int key, int pos, int lo, int keep) { return key <= pos && (key >= lo || key < keep); }

#define ATTN_BIAS_LEAD 256
#define ATTN_BIAS_TAIL 256
// a head's bias at distance 0 in the table (null: no bias)
__device__ __forceinline__ const float* attn_bias_row(const AttnOpts& opt, int head) {
    return opt.bias ? opt.bias + (size_t)head * (ATTN_BIAS_LEAD + opt.bias_n + ATTN_BIAS_TAIL) + ATTN_BIAS_LEAD : nullptr;
}
// the bias at a distance between -ATTN_BIAS_LEAD and bias_n - 1 + ATTN_BIAS_TAIL
__device__ __forceinline__ float attn_bias_at(const float* row, int distance) {
    return ZLM_CHK(row + distance, 4) ? __ldg(row + distance) : 0.f;
}

// a tile's raw dot products as base-2 exponents, dot * scale * log2(e), capped first where the mixer asks for it (tanh(y)
// through one exponential: 1 - 2 / (e^{2y} + 1), absolute error of a few 1e-7 of the cap).  Whether there is a cap is asked
// once for the tile (every thread of a launch answers alike), so a kernel without one pays a multiplication a score and
// nothing else
template <int NT> __device__ __forceinline__ void attn_scores_log2(float (&s)[NT][4], float scale_log2, float softcap) {
    if (softcap > 0.f) {
        const float k_in = 2.0f * scale_log2 / softcap, k_out = softcap * ATTN_LOG2E;         // 2^(dot * k_in) = e^{2y}
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[nt][e] = fmaf(-2.0f * k_out, __fdividef(1.0f, exp2f(s[nt][e] * k_in) + 1.0f), k_out);
    } else {
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[nt][e] *= scale_log2;
    }
}

// the running maximum a row starts from (base-2 exponent) when the softmax has a sink
__device__ __forceinline__ float attn_sink_log2(const float* sinks, int head) {
    return (sinks && ZLM_CHK(sinks + head, 4)) ? sinks[head] * 1.4426950408889634f : 0.f;
}

// element offset of (row, 16-byte chunk) inside a [64][HD] tile; rows of 128 bytes
// or more are swizzled so that ldmatrix reads 8 rows without bank conflicts
template <int HD> __device__ __forceinline__ int tile_off(int row, int chunk) {
    constexpr int SW = (HD % 64 == 0) ? 7 : 0;
    return row * HD + ((chunk ^ (row & SW)) << 3);
}

