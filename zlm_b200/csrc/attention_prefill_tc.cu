// Prefill attention on the 5th-generation tensor cores, bf16 paged cache: heads of 128, or keys of 192 with
// values of 128 (KD: the keys are then three slabs of 64 dims where a head of 128 has two; one head a block).
//
// A block owns 128 query tokens of one sequence and HPC (1 or 2) query heads of one kv
// group, and walks the keys these tokens may see in steps of 128 (two pages of the cache);
// the heads of a block share the K and V tiles in shared memory.
//   warp 0      TMA producer: the Q tiles once, then a ring of K steps and one of V steps
//   warp 1      issues every head's S = Q K^T (128 x 128, fp32 in tensor memory) and
//               O += P V (128 x 128 in tensor memory) with tcgen05.mma: the warp stays whole and
//               one elected lane issues the 8 products of a step from one block of instructions
//               (measured alone, such a block issues a product every 65 cycles, the tensor cores'
//               rate; a thread issuing them one by one needs 108 each, and two issuing warps
//               slow each other)
//   4 warps per head: softmax, thread = query row.  They take the row's 128 scores into
//               registers (and give S back: the next step's S is computed while this step's
//               softmax runs), mask by the row's own position and window, keep a running maximum
//               and sum in fp32, write P as bf16 into shared memory in the layout the second
//               product wants, and at the end scale O by 1/sum and store it.
// The running maximum is lazy: O is only rescaled (read from tensor memory, scaled,
// written back) when a row's maximum grows by more than 2^8; otherwise the old
// reference stays, which changes nothing in exact arithmetic (the same reference is
// used for P and for the sum) and keeps P below 2^8.
// A sequence with an odd number of pages loads its last page twice; the second copy's keys
// lie beyond every row's position and are masked.  Every wait is bounded (see gemm_tcgen05.cu).
//
// Options (AttnOpts, attn_common.cuh): keys of the query's own chunk of positions only; a tanh cap on the scores
// (a series of multiply-adds where a warp's scores of a step are all below half the cap; else tanh through one exponential
// and one reciprocal of the special-function unit, three such operations a score instead of one); a sink per query head; several key heads on one value head; the
// sequence's first keys beside a window; a bias by distance (heads of 128 only), read from the table where a step's
// distances differ and added as one number where they all read its last entry.
//
// Formula: s_t = (q . k_t) / sqrt(hd) for t in [t_start, pos], softmax, o = sum p_t v_t
// (src/kernels/transformer/attention.zig:86-164; per-row bound in block prefill:
// src/runtime/executor.zig:565-584; window start: :93-98).
#define TC_FAMILY 2
#include "tc_common.cuh"
#include "attn_common.cuh"
#include <math.h>

#define FA_BM 128          // query rows per block
#define FA_HD 128          // head size this kernel is built for
#define FA_BK 128          // keys per step: two pages
#define FA_RESCALE 8.0f    // log2 units
#define FA_THREADS(H) (64 + 128 * (H))      // producer, issuing warp, 4 softmax warps per head


// 2^x on the special-function unit; the arguments here are at most 2^8 after the lazy rescale
__device__ __forceinline__ float fa_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
// a raw score as a capped base-2 exponent: k_out * tanh(y), y = s * scale / softcap, with k_in = 2 * scale *
// log2(e) / softcap (so that 2^(s * k_in) = e^{2y}) and k_out = softcap * log2(e); tanh(y) = 1 - 2 / (e^{2y} + 1).
__device__ __forceinline__ float fa_cap(float s, float k_in, float k_out) {
    float r;
    asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(r) : "f"(fa_ex2(s * k_in) + 1.0f));
    return fmaf(-2.0f * k_out, r, k_out);
}
// two raw scores with |y| <= 1/2 as capped base-2 exponents: scale_log2 * s * (tanh(y) / y), the quotient by its Taylor
// series in y^2 (what is left out is below 1e-7); multiply-adds, where the form above keeps the special-function unit busy
__device__ __forceinline__ float2 fa_cap_small(float2 s, float k_y, float scale_log2) {
    const float2 y = __fmul2_rn(s, make_float2(k_y, k_y)), x = __fmul2_rn(y, y);
    float2 p = make_float2(21844.0f / 6081075.0f, 21844.0f / 6081075.0f);
    p = __ffma2_rn(p, x, make_float2(-1382.0f / 155925.0f, -1382.0f / 155925.0f));
    p = __ffma2_rn(p, x, make_float2(62.0f / 2835.0f, 62.0f / 2835.0f));
    p = __ffma2_rn(p, x, make_float2(-17.0f / 315.0f, -17.0f / 315.0f));
    p = __ffma2_rn(p, x, make_float2(2.0f / 15.0f, 2.0f / 15.0f));
    p = __ffma2_rn(p, x, make_float2(-1.0f / 3.0f, -1.0f / 3.0f));
    p = __ffma2_rn(p, x, make_float2(1.0f, 1.0f));
    return __fmul2_rn(__fmul2_rn(s, make_float2(scale_log2, scale_log2)), p);
}
__device__ __forceinline__ unsigned fa_pack(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *(unsigned*)&v;
}
// Eight products from one block of instructions, issued by one elected lane of a whole warp;
// descriptors count in units of 16 bytes.
// S = Q K^T over the head's 128 dims: both operands K-major in two halves of 64 dims, 16 KB
// apart (128 rows of 128 bytes); 16 dims are 32 bytes on.  The first product overwrites.
__device__ __forceinline__ void fa_issue_s8(unsigned tmem_d, uint64_t qd, uint64_t kd, unsigned idesc) {
    asm volatile(
        "{\n\t.reg .pred q, p0, p1;\n\t.reg .b64 da, db;\n\t"
        "elect.sync _|q, 0xffffffff;\n\t"
        "setp.ne.b32 p0, 0, 0;\n\tsetp.eq.b32 p1, 0, 0;\n\t"
        "@q tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p0;\n\t"
        "add.u64 da, %1, 2;\n\tadd.u64 db, %2, 2;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 4;\n\tadd.u64 db, %2, 4;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 6;\n\tadd.u64 db, %2, 6;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 1024;\n\tadd.u64 db, %2, 1024;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 1026;\n\tadd.u64 db, %2, 1026;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 1028;\n\tadd.u64 db, %2, 1028;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 1030;\n\tadd.u64 db, %2, 1030;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "}\n"
        ::"r"(tmem_d), "l"(qd), "l"(kd), "r"(idesc) : "memory");
}
// O (+)= P V over the step's 128 keys, 16 keys a product.  P K-major in two halves of 64 keys
// (16 KB apart; 16 keys are 32 bytes on); V MN-major, a page after the other (16 KB apart), 16
// keys are 2 KB on.  The first product accumulates unless it is the block's first step.
__device__ __forceinline__ void fa_issue_pv8(unsigned tmem_d, uint64_t pd, uint64_t vd, unsigned idesc, unsigned acc_first) {
    asm volatile(
        "{\n\t.reg .pred q, p0, p1;\n\t.reg .b64 da, db;\n\t"
        "elect.sync _|q, 0xffffffff;\n\t"
        "setp.ne.b32 p0, %4, 0;\n\tsetp.eq.b32 p1, 0, 0;\n\t"
        "@q tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p0;\n\t"
        "add.u64 da, %1, 2;\n\tadd.u64 db, %2, 128;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 4;\n\tadd.u64 db, %2, 256;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 6;\n\tadd.u64 db, %2, 384;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 1024;\n\tadd.u64 db, %2, 1024;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 1026;\n\tadd.u64 db, %2, 1152;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 1028;\n\tadd.u64 db, %2, 1280;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 1030;\n\tadd.u64 db, %2, 1408;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "}\n"
        ::"r"(tmem_d), "l"(pd), "l"(vd), "r"(idesc), "r"(acc_first) : "memory");
}
// four more products of S: a third slab of 64 dims, 32 KB beyond the first in both operands (keys of 192)
__device__ __forceinline__ void fa_issue_s4_more(unsigned tmem_d, uint64_t qd, uint64_t kd, unsigned idesc) {
    asm volatile(
        "{\n\t.reg .pred q, p1;\n\t.reg .b64 da, db;\n\t"
        "elect.sync _|q, 0xffffffff;\n\t"
        "setp.eq.b32 p1, 0, 0;\n\t"
        "add.u64 da, %1, 2048;\n\tadd.u64 db, %2, 2048;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 2050;\n\tadd.u64 db, %2, 2050;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 2052;\n\tadd.u64 db, %2, 2052;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "add.u64 da, %1, 2054;\n\tadd.u64 db, %2, 2054;\n\t@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p1;\n\t"
        "}\n"
        ::"r"(tmem_d), "l"(qd), "l"(kd), "r"(idesc) : "memory");
}
// an arrival at `bar` once the products issued so far have retired, from the same elected lane
__device__ __forceinline__ void fa_commit(uint64_t* bar) {
    asm volatile(
        "{\n\t.reg .pred q;\n\telect.sync _|q, 0xffffffff;\n\t"
        "@q tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n\t}\n" ::"r"(smem_u32(bar)) : "memory");
}

// CAP: built with the cap on the scores (the form without it keeps the plain softmax's registers)
// KD: the keys' and queries' width (128, or 192 with values of 128: rows of the pool and of q and out are KD wide)
// EXTRA: FA_BIAS, built with a bias by distance; FA_KEEP, with first keys kept beside the window (not both)
#define FA_PLAIN 0
#define FA_BIAS 1
#define FA_KEEP 2
template <int HPC, bool CAP, int KD = FA_HD, int EXTRA = FA_PLAIN>
__global__ void __launch_bounds__(FA_THREADS(HPC), 1)
attention_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv,
                            __nv_bfloat16* __restrict__ out, int out_stride, const int* __restrict__ block_table,
                            int table_stride, const int* __restrict__ cu_seqlens, const int* __restrict__ seq_slot,
                            const int* __restrict__ seq_start, int R, int tiles_per_seq, int nq, int nkv,
                            float scale_log2, int window, int sink, AttnOpts opt) {
    static_assert((KD == 128 || KD == 192) && (KD == 128 || HPC == 1), "keys of 128, or of 192 with one head a block");
    constexpr int NKH = KD / 64;                                    // slabs of 64 dims in a query or key row
    constexpr int KST = (HPC == 2 || KD > 128) ? 1 : 2;             // stages of keys and of values: what fits beside
    constexpr int VST = HPC == 2 ? 2 : 3;                           // the Q and P tiles (224 KB in all)
    constexpr unsigned SLAB = FA_BM * 64 * 2;                       // [128 rows][64 dims]
    constexpr unsigned Q_BYTES = NKH * SLAB;                        // slabs of [128][64]
    constexpr unsigned P_BYTES = FA_BM * FA_BK * 2;                 // two halves of [128 rows][64 keys]
    constexpr unsigned PAGE_BYTES = ZLM_PAGE * FA_HD * 2;           // V of one page: two halves of [64][64]
    constexpr unsigned KV_BYTES = 2 * PAGE_BYTES;                   // V of a step
    constexpr unsigned K_BYTES = NKH * SLAB;                        // K of a step: slabs of [128 keys][64 dims]
    static_assert(SLAB == 16384 && P_BYTES / 2 == 16384 && KV_BYTES / 2 == 16384 && PAGE_BYTES == 16384,
                  "the constants of the issue blocks");
    static_assert(HPC * (Q_BYTES + P_BYTES) + KST * K_BYTES + VST * KV_BYTES <= 7 * 32768, "the tiles' shared memory");
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = (unsigned char*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    unsigned char* sQ = smem;                                       // [HPC] Q tiles
    unsigned char* sP = sQ + HPC * Q_BYTES;                         // [HPC] P tiles
    unsigned char* sK = sP + HPC * P_BYTES;                         // [KST]: dims 0..63 of the 128 keys, then dims 64..127, ...
    unsigned char* sV = sK + KST * K_BYTES;                         // [VST]: page 0 (two halves), page 1
    uint64_t* q_full = (uint64_t*)(sV + VST * KV_BYTES);
    uint64_t* k_full = q_full + 1;             // [KST]      TMA bytes landed
    uint64_t* k_empty = k_full + KST;          // [KST]      the heads' S = Q K^T of that step retired
    uint64_t* v_full = k_empty + KST;          // [VST]
    uint64_t* v_empty = v_full + VST;          // [VST]      the heads' O += P V of that step retired
    uint64_t* s_full = v_empty + VST;          // [HPC]      S = Q K^T retired
    uint64_t* s_empty = s_full + HPC;          // [HPC]      the softmax warps have S in registers
    uint64_t* p_full = s_empty + HPC;          // [HPC]      P written (and O rescaled if needed)
    uint64_t* pv_done = p_full + HPC;          // [HPC]      O += P V of a step retired: P may be overwritten, O is at rest
    unsigned* tmem_slot = (unsigned*)(pv_done + HPC);
    volatile int* abort_flag = (volatile int*)(tmem_slot + 1);
    {
        // the tiles leave less than a kilobyte for rounding the base up to the 1024 bytes that the
        // swizzled tiles want; if that ever is not enough, the block says so and leaves
        unsigned dyn;
        asm volatile("mov.u32 %0, %%dynamic_smem_size;\n" : "=r"(dyn));
        if ((unsigned char*)(tmem_slot + 4) > smem_raw + dyn) {
            if (threadIdx.x == 0) zlm_report_status((TC_FAMILY << 8) | 0x40);
            return;
        }
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // blocks are numbered so that the tiles with the most pages (the last rows of the longest
    // prompts) start first and the short ones fill the gaps at the end
    const int n_hb = nq / HPC;                 // head groups
    const int rank = blockIdx.x / n_hb;        // 0 = the last tile of a sequence
    const int b = tiles_per_seq - 1 - rank / R, r = rank % R;
    const int head0 = (blockIdx.x % n_hb) * HPC;   // the block's first query head; its heads share a kv head
    if (!ZLM_CHK(cu_seqlens + r, 8) || !ZLM_CHK(seq_start + r, 4) || !ZLM_CHK(seq_slot + r, 4)) return;   // block-uniform
    const int tok0 = cu_seqlens[r], n_new = cu_seqlens[r + 1] - tok0;
    const int row0 = b * FA_BM;
    if (row0 >= n_new) return;
    const int rows = min(FA_BM, n_new - row0);
    const int kvh = head0 / (nq / nkv);
    const int start = seq_start[r];
    const int* pages = block_table + (size_t)seq_slot[r] * table_stride;
    const int first_pos = start + row0, last_pos = start + row0 + rows - 1;
    const int blk_lo = attn_first_key(first_pos, window, opt.chunk);
    const int last_lo = attn_first_key(last_pos, window, opt.chunk);        // (a row's first key does not fall as positions grow)
    const int page_heads = nkv + nkv / opt.v_share;                         // heads of [64][128] in a page: keys, then values
    const int page_hi = last_pos / ZLM_PAGE + 1;
    constexpr bool BIAS = EXTRA == FA_BIAS, KEEP = EXTRA == FA_KEEP;
    const AttnWalk walk(blk_lo / ZLM_PAGE, page_hi, KEEP ? opt.keep : 0);
    const int NS = (walk.n + 1) / 2;           // steps of two pages

    // K and V of step j into their stages (the producer thread; false if a wait gave up)
    int k_issued = 0, v_issued = 0;
    auto load_step = [&](int j) -> bool {
        int page[2];
#pragma unroll
        for (int pg = 0; pg < 2; ++pg) {
            // an odd last page comes twice: its second copy's keys are beyond every row's position
            const int lp = min(walk.page(2 * j + pg), page_hi - 1);
            page[pg] = ZLM_CHK(pages + lp, 4) ? pages[lp] : 0;
        }
        const int sk = j % KST, sv = j % VST;
        if (!mbar_wait(&k_empty[sk], ((j / KST) & 1) ^ 1, abort_flag, 1)) return false;
        mbar_expect_tx(&k_full[sk], K_BYTES);
#pragma unroll
        for (int pg = 0; pg < 2; ++pg) {
            // K: [slab][page][64 keys][64 dims]: the 128 keys of a slab are one operand tile
            const int krow = (page[pg] * page_heads + kvh) * ZLM_PAGE;
#pragma unroll
            for (int sl = 0; sl < NKH; ++sl)
                tma_load_2d(sK + sk * K_BYTES + sl * SLAB + pg * (SLAB / 2), &map_kv, 64 * sl, krow, &k_full[sk]);
        }
        k_issued = j + 1;
        if (!mbar_wait(&v_empty[sv], ((j / VST) & 1) ^ 1, abort_flag, 1)) return false;
        mbar_expect_tx(&v_full[sv], KV_BYTES);
#pragma unroll
        for (int pg = 0; pg < 2; ++pg) {
            // V: [page][half][64 keys][64 dims]
            const int vrow = (page[pg] * page_heads + nkv + kvh / opt.v_share) * ZLM_PAGE;
            tma_load_2d(sV + sv * KV_BYTES + pg * PAGE_BYTES, &map_kv, 0, vrow, &v_full[sv]);
            tma_load_2d(sV + sv * KV_BYTES + pg * PAGE_BYTES + PAGE_BYTES / 2, &map_kv, 64, vrow, &v_full[sv]);
        }
        v_issued = j + 1;
        return true;
    };
    if (threadIdx.x == 0) {
        asm volatile("prefetch.tensormap [%0];\n" ::"l"(&map_q) : "memory");
        asm volatile("prefetch.tensormap [%0];\n" ::"l"(&map_kv) : "memory");
        mbar_init(q_full, 1);
        for (int s = 0; s < KST; ++s) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); }
        for (int s = 0; s < VST; ++s) { mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1); }
        for (int i = 0; i < HPC; ++i) {
            mbar_init(&s_full[i], 1); mbar_init(&s_empty[i], 4); mbar_init(&p_full[i], 4); mbar_init(&pv_done[i], 1);
        }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
        // this thread is the producer: the Q tiles and the first step's keys and values are on
        // their way before the block has met (they arrive at barriers this thread has just set
        // up; their stages are free, so nothing waits).  Q and this step's keys and values come
        // from the kernel before: as a dependent launch the block is set up while that kernel
        // drains, and waits for it here.
        pdl_launch_dependents();
        pdl_wait();
        mbar_expect_tx(q_full, HPC * Q_BYTES);
        for (int h = 0; h < HPC; ++h) {
            // Q: slabs of 64 columns per head, 128 token rows
#pragma unroll
            for (int sl = 0; sl < NKH; ++sl)
                tma_load_2d(sQ + h * Q_BYTES + sl * SLAB, &map_q, (head0 + h) * KD + 64 * sl, tok0 + row0, q_full);
        }
        if (NS > 0) load_step(0);
    }
    if (warp == 1) {
        // columns per head: S [0,128), O [128,256)
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n"
                     ::"r"(smem_u32(tmem_slot)), "r"(256u * HPC) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    pdl_wait();              // (thread 0 has waited before the block met; for the others this returns at once)
    const unsigned tmem_base = *tmem_slot;

    if (warp == 0) {
        if (lane == 0) {
            for (int j = 1; j < NS; ++j)
                if (!load_step(j)) break;
            if (*abort_flag) {
                mbar_drain(q_full, 0);
                for (int j = max(0, k_issued - KST); j < k_issued; ++j) mbar_drain(&k_full[j % KST], (j / KST) & 1);
                for (int j = max(0, v_issued - VST); j < v_issued; ++j) mbar_drain(&v_full[j % VST], (j / VST) & 1);
            }
        }
    } else if (warp == 1) {
        // S: M 128, N 128, both operands K-major.  O: M 128, N 128, A (P) K-major, B (V) MN-major.
        const unsigned idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((unsigned)(FA_BK >> 3) << 17) | (8u << 24);
        const unsigned idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((unsigned)(FA_HD >> 3) << 17) | (8u << 24);
        bool ok = mbar_wait_warp(q_full, 0, abort_flag, 2);
        // S of step j for every head: the keys are there, and the head's softmax warps have taken
        // S of step j - 1 into registers
        auto issue_s = [&](int j) -> bool {
            const int s = j % KST;
            if (!mbar_wait_warp(&k_full[s], (j / KST) & 1, abort_flag, 2)) return false;
            const uint64_t kd = make_desc(smem_u32(sK + s * K_BYTES));
#pragma unroll
            for (int h = 0; h < HPC; ++h) {
                if (j > 0 && !mbar_wait_warp(&s_empty[h], (j - 1) & 1, abort_flag, 5)) return false;
                tc_fence_after();
                fa_issue_s8(tmem_base + h * 256, make_desc(smem_u32(sQ + h * Q_BYTES)), kd, idesc_s);
                if (KD > 128) fa_issue_s4_more(tmem_base + h * 256, make_desc(smem_u32(sQ + h * Q_BYTES)), kd, idesc_s);
                fa_commit(&s_full[h]);
            }
            fa_commit(&k_empty[s]);                // the keys' stage is free when the heads' S have retired
            return true;
        };
        if (ok && NS > 0) ok = issue_s(0);
        for (int j = 0; j < NS && ok; ++j) {
            if (j + 1 < NS) { ok = issue_s(j + 1); if (!ok) break; }
            const int s = j % VST;
            ok = mbar_wait_warp(&v_full[s], (j / VST) & 1, abort_flag, 2);
            if (!ok) break;
            // a V page: [64 keys][128 bytes] for dims 0..63, then the same for dims 64..127:
            // 16 keys a product = 2048 bytes; next 64 dims 8192 bytes on; 8-key groups 1024 bytes apart
            const uint64_t vd = make_desc_ex(smem_u32(sV + s * KV_BYTES), PAGE_BYTES / 2, 1024);
#pragma unroll
            for (int h = 0; h < HPC; ++h) {
                ok = mbar_wait_warp(&p_full[h], j & 1, abort_flag, 6);
                if (!ok) break;
                tc_fence_after();
                fa_issue_pv8(tmem_base + h * 256 + 128, make_desc(smem_u32(sP + h * P_BYTES)), vd, idesc_o, j != 0);
                fa_commit(&pv_done[h]);
            }
            if (!ok) break;
            fa_commit(&v_empty[s]);                // the values' stage is free when the heads' products have retired
        }
        if (!ok) {
            for (int h = 0; h < HPC; ++h) {        // let the softmax warps out
                fa_commit(&s_full[h]);
                fa_commit(&pv_done[h]);
            }
        }
    } else {
        const int hh = (warp - 2) >> 2;                 // which of the block's heads this warp serves
        const int head = head0 + hh;
        const unsigned tmem_s = tmem_base + hh * 256, tmem_o = tmem_s + 128;
        unsigned char* const sP_h = sP + hh * P_BYTES;
        const int lg = warp & 3;
        const int i = lg * 32 + lane;                   // row of the tile = lane of tensor memory
        const bool row_ok = i < rows;
        const int pos = start + row0 + i;
        const int lo = attn_first_key(pos, window, opt.chunk);
        const unsigned lane_addr = (unsigned)(lg * 32) << 16;
        // (sink: a key of score 0, or sinks[head], without a value, one more term in the row's sum)
        float m_ref = sink ? attn_sink_log2(opt.sinks, head) : -INFINITY, l = sink ? 1.f : 0.f;
        constexpr bool capped = CAP;
        const int keep = KEEP ? opt.keep : 0;
        const float* brow = BIAS ? attn_bias_row(opt, head) : nullptr;
        const float far_bias = BIAS ? attn_bias_at(brow, opt.bias_n - 1) * ATTN_LOG2E : 0.f;
        constexpr bool final_scores = CAP || BIAS;      // the scores become base-2 exponents before their maximum is taken
        const float k_in = capped ? 2.0f * scale_log2 / opt.softcap : 0.f, k_out = opt.softcap * ATTN_LOG2E;
        const float k_y = k_in * (0.5f / ATTN_LOG2E);                // y = s * k_y
        bool ok = true;
        for (int j = 0; j < NS; ++j) {
            ok = mbar_wait_warp(&s_full[hh], j & 1, abort_flag, 3);
            tc_fence_after();
            if (!ok || *abort_flag) { ok = false; break; }
            // the step's two pages need not be neighbours: the kept ones lie before the window's
            const int kb0 = (KEEP ? walk.page(2 * j) : walk.lo + 2 * j) * ZLM_PAGE, kb1 = KEEP ? walk.page(2 * j + 1) * ZLM_PAGE : kb0 + ZLM_PAGE;
            // a step that every row of the tile sees whole needs no mask (block-uniform test)
            const bool inner = rows == FA_BM && kb1 + ZLM_PAGE - 1 <= first_pos && kb0 >= last_lo;
            // the row's 128 scores into registers in one round trip to tensor memory; then S is free
            float sv[FA_BK];
#pragma unroll
            for (int c = 0; c < FA_BK; c += 16) tc_ld16_nowait(tmem_s + lane_addr + c, sv + c);
            tc_wait_ld();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&s_empty[hh]);
            if (capped) {
                float am[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int e = 0; e < FA_BK; ++e) am[e & 3] = fmaxf(am[e & 3], fabsf(sv[e]));
                if (__all_sync(0xffffffffu, fmaxf(fmaxf(am[0], am[1]), fmaxf(am[2], am[3])) * k_y <= 0.5f)) {
#pragma unroll
                    for (int e = 0; e < FA_BK; e += 2) {
                        const float2 r = fa_cap_small(make_float2(sv[e], sv[e + 1]), k_y, scale_log2);
                        sv[e] = r.x;
                        sv[e + 1] = r.y;
                    }
                } else {
#pragma unroll
                    for (int e = 0; e < FA_BK; ++e) sv[e] = fa_cap(sv[e], k_in, k_out);
                }
            } else if (BIAS) {
#pragma unroll
                for (int e = 0; e < FA_BK; ++e) sv[e] *= scale_log2;
            }
            // (where the step's distances all read the bias table's last number, that one is part of the reference)
            const bool near = BIAS && first_pos - (kb1 + ZLM_PAGE - 1) < opt.bias_n - 1;        // block-uniform
            if (near) {
#pragma unroll
                for (int e = 0; e < FA_BK; ++e)           // (neighbouring rows read neighbouring numbers)
                    sv[e] = fmaf(attn_bias_at(brow + (pos - kb0), -e), ATTN_LOG2E, sv[e]);
            }
            // four independent chains of maxima (raw scores without cap and bias; the scale is positive)
            float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
            if (inner) {
#pragma unroll
                for (int e = 0; e < FA_BK; ++e) mx4[e & 3] = fmaxf(mx4[e & 3], sv[e]);
            } else {
#pragma unroll
                for (int e = 0; e < FA_BK; ++e) {
                    const int key = (!KEEP || e < ZLM_PAGE ? kb0 : kb1 - ZLM_PAGE) + e;
                    const bool vis = row_ok && (KEEP ? attn_sees(key, pos, lo, keep) : key <= pos && key >= lo);
                    sv[e] = vis ? sv[e] : -INFINITY;
                    mx4[e & 3] = fmaxf(mx4[e & 3], sv[e]);
                }
            }
            const float mx_raw = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
            const float mx = final_scores ? mx_raw + (BIAS && !near ? far_bias : 0.f) : mx_raw * scale_log2;          // -inf stays -inf
            // lazy reference: move it only when the maximum grew by more than 2^8
            const bool grow = mx > m_ref + FA_RESCALE;              // also true for the first real maximum
            const float m_new = grow ? mx : m_ref;
            const float alpha = (grow && m_ref != -INFINITY) ? exp2f(m_ref - m_new) : 1.0f;
            const bool need_rescale = grow && m_ref != -INFINITY && j > 0;
            // the product of step j - 1 has retired: its P may be overwritten, and O is at rest
            // (step j's cannot have been issued, it waits for this warp)
            if (j > 0) {
                ok = mbar_wait_warp(&pv_done[hh], (j - 1) & 1, abort_flag, 7);
                tc_fence_after();
                if (!ok) break;
            }
            if (__any_sync(0xffffffffu, need_rescale)) {
#pragma unroll 1
                for (int c = 0; c < FA_HD; c += 16) {
                    float ov[16];
                    tc_ld16(tmem_o + lane_addr + c, ov);
#pragma unroll
                    for (int e = 0; e < 16; ++e) ov[e] *= alpha;
                    tc_st16(tmem_o + lane_addr + c, ov);
                }
                tc_wait_st();
                tc_fence_before();
            }
            l *= alpha;
            m_ref = m_new;
            const float ref = (m_ref == -INFINITY ? 0.f : m_ref) - (BIAS && !near ? far_bias : 0.f);
            // P = 2^(s * scale - ref) (2^-inf = 0 for masked keys) -> shared memory: two halves of 64
            // keys, 128 bytes a row, 16-byte chunks swizzled by (row % 8)
            float ps4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int ch = 0; ch < FA_BK / 8; ++ch) {
                float p[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    p[e] = final_scores ? fa_ex2(sv[ch * 8 + e] - ref) : fa_ex2(fmaf(sv[ch * 8 + e], scale_log2, -ref));
                    ps4[e & 3] += p[e];
                }
                uint4 pk;
                pk.x = fa_pack(p[0], p[1]); pk.y = fa_pack(p[2], p[3]);
                pk.z = fa_pack(p[4], p[5]); pk.w = fa_pack(p[6], p[7]);
                *(uint4*)(sP_h + (ch >> 3) * (P_BYTES / 2) + i * 128 + (((ch & 7) ^ (i & 7)) << 4)) = pk;
            }
            l += (ps4[0] + ps4[1]) + (ps4[2] + ps4[3]);
            fence_async_smem();
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full[hh]);
        }
        if (ok && NS > 0) ok = mbar_wait_warp(&pv_done[hh], (NS - 1) & 1, abort_flag, 8);
        tc_fence_after();
        if (ok && !*abort_flag) {
            const float inv = row_ok ? 1.0f / l : 0.f;
            __nv_bfloat16* orow = out + (size_t)(tok0 + row0 + i) * out_stride + (size_t)head * KD;
#pragma unroll 1
            for (int c = 0; c < FA_HD; c += 16) {
                float ov[16];
                tc_ld16(tmem_o + lane_addr + c, ov);
                if (row_ok && ZLM_CHK(orow + c, 32)) {
                    uint4 a, bq;
                    a.x = fa_pack(ov[0] * inv, ov[1] * inv); a.y = fa_pack(ov[2] * inv, ov[3] * inv);
                    a.z = fa_pack(ov[4] * inv, ov[5] * inv); a.w = fa_pack(ov[6] * inv, ov[7] * inv);
                    bq.x = fa_pack(ov[8] * inv, ov[9] * inv); bq.y = fa_pack(ov[10] * inv, ov[11] * inv);
                    bq.z = fa_pack(ov[12] * inv, ov[13] * inv); bq.w = fa_pack(ov[14] * inv, ov[15] * inv);
                    *(uint4*)(orow + c) = a;
                    *(uint4*)(orow + c + 8) = bq;
                }
            }
            // (out's rows are as wide as the keys: the columns beyond the values become zeros)
            if (KD > FA_HD && row_ok && ZLM_CHK(orow + FA_HD, (KD - FA_HD) * 2)) {
#pragma unroll
                for (int c = FA_HD; c < KD; c += 8) *(uint4*)(orow + c) = make_uint4(0u, 0u, 0u, 0u);
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        __syncwarp();
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem_base), "r"(256u * HPC) : "memory");
    }
}

extern "C" int zlm_attention_prefill_tc_supported(int nq, int nkv, int hd, int q_stride, int out_stride) {
    return (hd == FA_HD && nkv > 0 && nq % nkv == 0 && q_stride % 8 == 0 && out_stride % 8 == 0) ? 1 : 0;
}
// the same for keys of `hd` with values of `vd` columns (the rows of the pool, of q and of out are hd wide)
extern "C" int zlm_attention_prefill_tc_vd_supported(int nq, int nkv, int hd, int vd, int q_stride, int out_stride) {
    if (vd == hd) return zlm_attention_prefill_tc_supported(nq, nkv, hd, q_stride, out_stride);
    return (hd == 192 && vd == FA_HD && nkv > 0 && nq % nkv == 0 && q_stride % 8 == 0 && out_stride % 8 == 0) ? 1 : 0;
}

// pool_rows: pages * 2 * nkv * 64 (all rows of the layer's pool, head size 128 each)
static int g_fa_heads = 0;

// Heads of a kv group per block.  Two heads can share a block (they share its keys and values,
// and one head's softmax runs beside the other's: a step of 128 keys takes the two about 4,000
// cycles against 2,500 for one alone), but the blocks are then half as many and the longest
// 1.6 times as long.  The step takes about as long as the larger of its longest block (the last
// tile of the longest prompt) and its whole work spread over the SMs; the form for which that is
// smaller runs (2,048 tokens, 16 heads over 8: 38 us with one head a block, 46 with two; 32 over
// 8: 73 and 54).  Odd groups take one.
extern "C" int zlm_attention_prefill_tc_heads(int R, int max_new, int nq, int nkv) {
    if (nkv <= 0 || nq % nkv != 0 || (nq / nkv) % 2 != 0) return 1;
    if (g_fa_heads) return g_fa_heads;
    static int sms = 0;
    if (!sms) {
        int dev = 0;
        if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms <= 0)
            sms = 148;
    }
    const int tiles = (max_new + FA_BM - 1) / FA_BM;
    const double pairs_cost = 1.6;                                          // a block of two heads, per step, against one head
    const double work = (double)R * tiles * (tiles + 1) / 2 / sms;          // tiles' pages summed, per SM and head
    const double two = fmax(tiles * pairs_cost, work * (nq / 2) * pairs_cost), one = fmax((double)tiles, work * nq);
    return two <= one ? 2 : 1;
}

// vd: the values' columns (hd, or 128 under keys of 192: out's columns from vd on become zeros)
extern "C" int zlm_attention_prefill_tc_vd(void* out, int out_stride, const void* q, int q_stride, int T,
                                           const void* pool, long long pool_pages, const int* block_table,
                                           int table_stride, const int* cu_seqlens, const int* seq_slot,
                                           const int* seq_start, int R, int max_new, int nq, int nkv, int hd, int vd,
                                           float scale, int window, int sink, int chunk, float softcap, const float* sinks,
                                           int v_share, int keep, const float* bias, int bias_n, cudaStream_t st) {
    if (R == 0 || max_new == 0) return ZLM_OK;
    ZLM_REQUIRE_ATTN_OPTS("attention_prefill_tc");
    ZLM_REQUIRE(!(bias && keep) && (hd == FA_HD || !(bias || keep)), "attention_prefill_tc: a bias by distance and kept keys are built for heads of %d, one of them at a time", FA_HD);
    const AttnOpts opt{chunk, softcap, sinks, v_share, keep, bias, bias_n};
    const long long page_heads = nkv + nkv / v_share;
    ZLM_REQUIRE(zlm_attention_prefill_tc_vd_supported(nq, nkv, hd, vd, q_stride, out_stride),
                "attention_prefill_tc: %d heads over %d kv heads of size %d, values of %d (strides %d, %d) is not a shape this kernel takes",
                nq, nkv, hd, vd, q_stride, out_stride);
    ZLM_REQUIRE(((uintptr_t)q % 16 == 0) && ((uintptr_t)out % 16 == 0) && ((uintptr_t)pool % 16 == 0),
                "attention_prefill_tc: q, out and the pool must be 16-byte aligned");
    ZLM_REQUIRE(pool_pages * page_heads * ZLM_PAGE < 2147483647LL, "attention_prefill_tc: the pool has too many rows for a tensor map coordinate");
    CUtensorMap mq, mkv;
    int rc = zlm_make_map_2d(&mq, q, T, nq * hd, q_stride, FA_BM, 64);
    if (rc) return rc;
    rc = zlm_make_map_2d(&mkv, pool, pool_pages * page_heads * ZLM_PAGE, hd, hd, ZLM_PAGE, 64);
    if (rc) return rc;
    const int tiles = (max_new + FA_BM - 1) / FA_BM;
    const int hpc = hd > FA_HD ? 1 : zlm_attention_prefill_tc_heads(R, max_new, nq, nkv);
    ZLM_REQUIRE((long long)R * tiles * nq < 2147483647LL, "attention_prefill_tc: too many tiles");
    // seven tiles of 32 KB (Q and P per head, the K and V stages), barriers, and what is left of a kilobyte for rounding the base up
    size_t smem = (size_t)7 * FA_BK * FA_HD * 2 + 256 + 1024;
    if (smem > 232448) smem = 232448;
#define ZLM_FA_LAUNCH(H, C, KD, B)                                                                                  \
    {                                                                                                             \
        static bool attr_set_dev[64] = {}; bool& attr_set = attr_set_dev[zlm_device_index()];                     \
        if (!attr_set) {                                                                                          \
            cudaError_t e = cudaFuncSetAttribute(attention_prefill_tc_kernel<H, C, KD, B>,                           \
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);         \
            if (e != cudaSuccess) {                                                                               \
                zlm_set_error("attention_prefill_tc: cannot reserve %zu bytes of shared memory: %s", smem,        \
                              cudaGetErrorString(e));                                                             \
                return ZLM_ERR_CUDA;                                                                              \
            }                                                                                                     \
            attr_set = true;                                                                                      \
        }                                                                                                         \
        zlm_launch(attention_prefill_tc_kernel<H, C, KD, B>, dim3(R * tiles * (nq / H)), dim3(FA_THREADS(H)), smem, st, mq, mkv, \
                   (__nv_bfloat16*)out, out_stride, block_table, table_stride, cu_seqlens, seq_slot, seq_start,   \
                   R, tiles, nq, nkv, scale * 1.4426950408889634f, window, sink, opt);                                       \
    }
#define ZLM_FA_FORMS(X)                                                                                           \
    if (softcap > 0.f) {                                                                                          \
        if (hpc == 2) ZLM_FA_LAUNCH(2, true, FA_HD, X)                                                            \
        else ZLM_FA_LAUNCH(1, true, FA_HD, X)                                                                     \
    } else {                                                                                                      \
        if (hpc == 2) ZLM_FA_LAUNCH(2, false, FA_HD, X)                                                           \
        else ZLM_FA_LAUNCH(1, false, FA_HD, X)                                                                    \
    }
    if (hd > FA_HD) {
        if (softcap > 0.f) ZLM_FA_LAUNCH(1, true, 192, FA_PLAIN)
        else ZLM_FA_LAUNCH(1, false, 192, FA_PLAIN)
    } else if (bias) {
        ZLM_FA_FORMS(FA_BIAS)
    } else if (keep) {
        ZLM_FA_FORMS(FA_KEEP)
    } else {
        ZLM_FA_FORMS(FA_PLAIN)
    }
#undef ZLM_FA_FORMS
#undef ZLM_FA_LAUNCH
    return zlm_check_launch("attention_prefill_tc");
}

extern "C" int zlm_attention_prefill_tc(void* out, int out_stride, const void* q, int q_stride, int T,
                                        const void* pool, long long pool_pages, const int* block_table,
                                        int table_stride, const int* cu_seqlens, const int* seq_slot,
                                        const int* seq_start, int R, int max_new, int nq, int nkv, int hd,
                                        float scale, int window, int sink, int chunk, float softcap, const float* sinks,
                                        int v_share, int keep, const float* bias, int bias_n, cudaStream_t st) {
    return zlm_attention_prefill_tc_vd(out, out_stride, q, q_stride, T, pool, pool_pages, block_table, table_stride,
                                       cu_seqlens, seq_slot, seq_start, R, max_new, nq, nkv, hd, hd, scale, window, sink,
                                       chunk, softcap, sinks, v_share, keep, bias, bias_n, st);
}

// heads of a kv group per block: 0 lets the dispatcher choose; 1 or 2 force that many where the kv
// groups are even (odd groups always take one).  For tests and measurements.
extern "C" int zlm_attention_prefill_tc_set_heads(int heads) {
    ZLM_REQUIRE(heads >= 0 && heads <= 2, "attention_prefill_tc: %d heads per block cannot be forced", heads);
    g_fa_heads = heads;
    return ZLM_OK;
}

ZLM_TRANSLATION_UNIT(attention_prefill_tc)
