// Prefill attention over the paged bf16 cache: tiles of 64 query tokens of one
// sequence and one query head attend the sequence's keys page by page (a page is
// the 64-key tile), with the keys and values of the step's own tokens already in
// the cache.  S = Q K^T and O += P V run on the warp-level tensor cores; the
// running maximum and sum of the softmax are fp32; pages are staged with cp.async,
// double buffered.  Causality and the window are bounds on the key index per
// query row, so a chunk of a prompt attends the earlier chunks exactly as a whole
// prompt would.
//
// Options (AttnOpts, attn_common.cuh): keys of the query's own chunk of positions only, a tanh cap on the
// scores, a sink per query head in the softmax's denominator, several key heads on one value head, the sequence's first
// keys beside a window, a bias by distance.
//
// Formula: s_t = (q . k_t) / sqrt(hd) for t in [t_start, pos], softmax, o = sum
// p_t v_t (src/kernels/transformer/attention.zig:86-164); per-row bound in block
// prefill: src/runtime/executor.zig:565-584; window start: :93-98.
#include "attn_common.cuh"

#define PRE_BM 64
#define PRE_WARPS 4
#define PRE_THREADS (PRE_WARPS * 32)

// VD: how many of the HD value columns are used (a multiple of 16; the pool's values are HD wide, columns from VD
// on are padding that is neither loaded nor multiplied, and the output's columns from VD on are written as zeros)
template <int HD, int VD>
__global__ void __launch_bounds__(PRE_THREADS)
attention_prefill_kernel(__nv_bfloat16* __restrict__ out, int out_stride, const __nv_bfloat16* __restrict__ q,
                         int q_stride, const __nv_bfloat16* __restrict__ pool,
                         const int* __restrict__ block_table, int table_stride,
                         const int* __restrict__ cu_seqlens, const int* __restrict__ seq_slot,
                         const int* __restrict__ seq_start, int tiles_per_seq, int nq, int nkv,
                         float scale_log2, int window, int sink, AttnOpts opt) {
    constexpr int KS = HD / 16;
    constexpr int VS = VD / 16;
    constexpr int CH = HD / 8;
    constexpr int VCH = VD / 8;
    constexpr int TILE = ZLM_PAGE * HD;
    static_assert(VD % 16 == 0 && VD >= 16 && VD <= HD, "value columns");
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __nv_bfloat16* Ks = (__nv_bfloat16*)smem_raw;          // [2][TILE]
    __nv_bfloat16* Vs = Ks + 2 * TILE;                     // [2][TILE]

    const int r = blockIdx.x / tiles_per_seq, b = blockIdx.x % tiles_per_seq;
    const int head = blockIdx.y;
    if (!ZLM_CHK(cu_seqlens + r, 8) || !ZLM_CHK(seq_start + r, 4) || !ZLM_CHK(seq_slot + r, 4)) return;   // block-uniform
    const int tok0 = cu_seqlens[r], n_new = cu_seqlens[r + 1] - tok0;
    const int row0 = b * PRE_BM;
    if (row0 >= n_new) return;
    const int rows = min(PRE_BM, n_new - row0);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int g = lane >> 2, qd = lane & 3;
    const int kvh = head / (nq / nkv);
    const int start = seq_start[r];
    const int* pages = block_table + (size_t)seq_slot[r] * table_stride;
    const size_t page_stride = (size_t)(nkv + nkv / opt.v_share) * TILE;
    const size_t v_off = (size_t)(nkv - kvh + kvh / opt.v_share) * TILE;      // from this key head to its value head
    const int chunk = opt.chunk;
    const float softcap = opt.softcap;

    // positions of this thread's two rows; rows beyond the tile's tokens are idle
    const int i0 = warp * 16 + g, i1 = i0 + 8;
    bool ok0 = i0 < rows, ok1 = i1 < rows;
#ifdef ZLM_BOUNDS_CHECK
    // a row whose query or output lies outside the tensors passed is treated as idle
    ok0 = ok0 && ZLM_CHK(q + (size_t)(tok0 + row0 + i0) * q_stride + (size_t)head * HD, HD * 2) &&
          ZLM_CHK(out + (size_t)(tok0 + row0 + i0) * out_stride + (size_t)head * HD, HD * 2);
    ok1 = ok1 && ZLM_CHK(q + (size_t)(tok0 + row0 + i1) * q_stride + (size_t)head * HD, HD * 2) &&
          ZLM_CHK(out + (size_t)(tok0 + row0 + i1) * out_stride + (size_t)head * HD, HD * 2);
#endif
    const int pos0 = start + row0 + i0, pos1 = start + row0 + i1;
    const int lo0 = attn_first_key(pos0, window, chunk), lo1 = attn_first_key(pos1, window, chunk);
    // keys the block and this warp can need
    const int blk_first = start + row0, blk_last = start + row0 + rows - 1;
    const int blk_lo = attn_first_key(blk_first, window, chunk);
    const AttnWalk walk(blk_lo / ZLM_PAGE, blk_last / ZLM_PAGE + 1, opt.keep);
    const int keep = opt.keep;
    const float* brow = attn_bias_row(opt, head);
    const float far_bias = brow ? attn_bias_at(brow, opt.bias_n - 1) * ATTN_LOG2E : 0.f;
    const int w_first = start + row0 + warp * 16;
    const int w_last = min(blk_last, w_first + 15);
    const int w_lo = attn_first_key(w_first, window, chunk);
    const int w_last_lo = attn_first_key(w_last, window, chunk);        // (a row's first key does not fall as positions grow)
    const bool warp_idle = warp * 16 >= rows;

    unsigned qf[KS][4];
    {
        const __nv_bfloat16* q0 = q + (size_t)(tok0 + row0 + i0) * q_stride + (size_t)head * HD;
        const __nv_bfloat16* q1 = q + (size_t)(tok0 + row0 + i1) * q_stride + (size_t)head * HD;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            const int c = ks * 16 + qd * 2;
            qf[ks][0] = ok0 ? *(const unsigned*)(q0 + c) : 0u;
            qf[ks][1] = ok1 ? *(const unsigned*)(q1 + c) : 0u;
            qf[ks][2] = ok0 ? *(const unsigned*)(q0 + c + 8) : 0u;
            qf[ks][3] = ok1 ? *(const unsigned*)(q1 + c + 8) : 0u;
        }
    }
    float o[2 * VS][4];
#pragma unroll
    for (int i = 0; i < 2 * VS; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    if (sink) {          // a key of score 0 (or sinks[head]) without a value: one more term in every row's sum
        m0 = m1 = attn_sink_log2(opt.sinks, head);
        if (qd == 0) l0 = l1 = 1.f;
    }

    auto load_page = [&](int w, int stage) {
        const int p = walk.page(w);
        if (!ZLM_CHK(pages + p, 4)) return;
        const __nv_bfloat16* kb = pool + (size_t)pages[p] * page_stride + (size_t)kvh * TILE;
        const __nv_bfloat16* vb = kb + v_off;
        __nv_bfloat16* ks_ = Ks + stage * TILE;
        __nv_bfloat16* vs_ = Vs + stage * TILE;
        for (int id = tid; id < ZLM_PAGE * CH; id += PRE_THREADS) {
            const int rr = id / CH, c = id % CH;
            dec_cp_async16(ks_ + tile_off<HD>(rr, c), kb + rr * HD + c * 8);
            if (c < VCH) dec_cp_async16(vs_ + tile_off<HD>(rr, c), vb + rr * HD + c * 8);
        }
    };

    load_page(0, 0);
    dec_commit();
    for (int p = 0; p < walk.n; ++p) {
        const int stage = p & 1;
        dec_wait<0>();
        __syncthreads();
        if (p + 1 < walk.n) load_page(p + 1, stage ^ 1);
        dec_commit();
        const int kbase = walk.page(p) * ZLM_PAGE;
        if (warp_idle || kbase > w_last || (kbase + ZLM_PAGE - 1 < w_lo && kbase >= keep)) continue;   // warp-uniform
        const __nv_bfloat16* kt = Ks + stage * TILE;
        const __nv_bfloat16* vt = Vs + stage * TILE;

        float s[8][4];
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[nt][e] = 0.f;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
#pragma unroll
            for (int np = 0; np < 4; ++np) {           // pairs of key tiles
                const int mi = lane >> 3;
                const int row = np * 16 + (mi >> 1) * 8 + (lane & 7);
                const int col = ks * 2 + (mi & 1);
                unsigned b00, b01, b10, b11;
                dec_ldsm4(b00, b01, b10, b11, kt + tile_off<HD>(row, col));
                dec_mma(s[2 * np], qf[ks], b00, b01);
                dec_mma(s[2 * np + 1], qf[ks], b10, b11);
            }
        }
        // scale, mask by each row's own bounds, running maximum
        const bool edge = kbase + ZLM_PAGE - 1 > w_first || kbase < w_last_lo;
        float mx0 = -INFINITY, mx1 = -INFINITY;
        attn_scores_log2<8>(s, scale_log2, softcap);
        if (brow) {
            const bool far = w_first - (kbase + ZLM_PAGE - 1) >= opt.bias_n - 1;        // every distance reads the table's last entry
#pragma unroll
            for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int key = kbase + nt * 8 + qd * 2 + e;
                    s[nt][e] = far ? s[nt][e] + far_bias : fmaf(attn_bias_at(brow, pos0 - key), ATTN_LOG2E, s[nt][e]);
                    s[nt][2 + e] = far ? s[nt][2 + e] + far_bias : fmaf(attn_bias_at(brow, pos1 - key), ATTN_LOG2E, s[nt][2 + e]);
                }
        }
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int key = kbase + nt * 8 + qd * 2 + e;
                const bool a = !edge || attn_sees(key, pos0, lo0, keep);
                const bool c = !edge || attn_sees(key, pos1, lo1, keep);
                s[nt][e] = (a && ok0) ? s[nt][e] : -INFINITY;
                s[nt][2 + e] = (c && ok1) ? s[nt][2 + e] : -INFINITY;
                mx0 = fmaxf(mx0, s[nt][e]);
                mx1 = fmaxf(mx1, s[nt][2 + e]);
            }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);
        // a row that has seen no key yet keeps max = -inf; use 0 as its reference
        const float r0 = mn0 == -INFINITY ? 0.f : mn0, r1 = mn1 == -INFINITY ? 0.f : mn1;
        const float a0 = m0 == -INFINITY ? 0.f : exp2f(m0 - r0);
        const float a1 = m1 == -INFINITY ? 0.f : exp2f(m1 - r1);
        m0 = mn0;
        m1 = mn1;
        float ps0 = 0.f, ps1 = 0.f;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                s[nt][e] = exp2f(s[nt][e] - r0);             // exp2(-inf) = 0 for masked keys
                s[nt][2 + e] = exp2f(s[nt][2 + e] - r1);
                ps0 += s[nt][e];
                ps1 += s[nt][2 + e];
            }
        l0 = l0 * a0 + ps0;
        l1 = l1 * a1 + ps1;
#pragma unroll
        for (int i = 0; i < 2 * VS; ++i) {
            o[i][0] *= a0; o[i][1] *= a0; o[i][2] *= a1; o[i][3] *= a1;
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {               // 16 keys at a time
            unsigned pa[4];
            pa[0] = pack_bf16(s[2 * kk][0], s[2 * kk][1]);
            pa[1] = pack_bf16(s[2 * kk][2], s[2 * kk][3]);
            pa[2] = pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]);
            pa[3] = pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3]);
#pragma unroll
            for (int dn = 0; dn < VS; ++dn) {
                const int mi = lane >> 3;
                const int row = kk * 16 + (mi & 1) * 8 + (lane & 7);
                const int col = dn * 2 + (mi >> 1);
                unsigned b0, b1, b2, b3;
                dec_ldsm4t(b0, b1, b2, b3, vt + tile_off<HD>(row, col));
                dec_mma(o[2 * dn], pa, b0, b1);
                dec_mma(o[2 * dn + 1], pa, b2, b3);
            }
        }
    }
    dec_wait<0>();

    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    const float inv0 = ok0 ? 1.0f / l0 : 0.f, inv1 = ok1 ? 1.0f / l1 : 0.f;
    __nv_bfloat16* o0 = out + (size_t)(tok0 + row0 + i0) * out_stride + (size_t)head * HD;
    __nv_bfloat16* o1 = out + (size_t)(tok0 + row0 + i1) * out_stride + (size_t)head * HD;
#pragma unroll
    for (int i = 0; i < 2 * VS; ++i) {
        const int d = i * 8 + qd * 2;
        if (ok0) *(unsigned*)(o0 + d) = pack_bf16(o[i][0] * inv0, o[i][1] * inv0);
        if (ok1) *(unsigned*)(o1 + d) = pack_bf16(o[i][2] * inv1, o[i][3] * inv1);
    }
#pragma unroll
    for (int i = 2 * VS; i < 2 * KS; ++i) {
        const int d = i * 8 + qd * 2;
        if (ok0) *(unsigned*)(o0 + d) = 0u;
        if (ok1) *(unsigned*)(o1 + d) = 0u;
    }
}

template <int HD, int VD = HD>
static int launch_prefill(__nv_bfloat16* out, int out_stride, const __nv_bfloat16* q, int q_stride,
                          const __nv_bfloat16* pool, const int* block_table, int table_stride,
                          const int* cu_seqlens, const int* seq_slot, const int* seq_start, int R, int max_new,
                          int nq, int nkv, float scale, int window, int sink, AttnOpts opt, cudaStream_t st) {
    const size_t smem = (size_t)4 * ZLM_PAGE * HD * sizeof(__nv_bfloat16);
    auto kern = attention_prefill_kernel<HD, VD>;
    static bool attr_set_dev[64] = {}; bool& attr_set = attr_set_dev[zlm_device_index()];
    if (!attr_set) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) {
            zlm_set_error("attention_prefill: cannot reserve %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
            return ZLM_ERR_CUDA;
        }
        attr_set = true;
    }
    const int tiles = (max_new + PRE_BM - 1) / PRE_BM;
    ZLM_REQUIRE((long long)R * tiles < 2147483647LL && nq <= 65535, "attention_prefill: too many tiles");
    dim3 grid(R * tiles, nq);
    kern<<<grid, PRE_THREADS, smem, st>>>(out, out_stride, q, q_stride, pool, block_table, table_stride, cu_seqlens,
                                         seq_slot, seq_start, tiles, nq, nkv, scale * 1.4426950408889634f, window, sink, opt);
    return zlm_check_launch("attention_prefill");
}

extern "C" int zlm_attention_prefill_supported(int nq, int nkv, int hd) {
    return (nkv > 0 && nq % nkv == 0 && hd % 16 == 0 && hd >= 16 && hd <= 192) ? 1 : 0;
}

// q tokens are packed by sequence: sequence r owns tokens cu_seqlens[r] .. cu_seqlens[r+1]-1 at positions
// seq_start[r] .. of slot seq_slot[r]; max_new is the largest token count of a sequence
extern "C" int zlm_attention_prefill(void* out, int out_stride, const void* q, int q_stride, const void* pool,
                                     const int* block_table, int table_stride, const int* cu_seqlens,
                                     const int* seq_slot, const int* seq_start, int R, int max_new, int nq,
                                     int nkv, int hd, float scale, int window, int sink, int chunk, float softcap,
                                     const float* sinks, int v_share, int keep, const float* bias, int bias_n, cudaStream_t st) {
    if (R == 0 || max_new == 0) return ZLM_OK;
    ZLM_REQUIRE(zlm_attention_prefill_supported(nq, nkv, hd),
                "attention_prefill: %d heads over %d kv heads of size %d is not a shape this kernel takes", nq, nkv, hd);
    ZLM_REQUIRE_ATTN_OPTS("attention_prefill");
    const AttnOpts opt{chunk, softcap, sinks, v_share, keep, bias, bias_n};
    ZLM_REQUIRE(q_stride % 2 == 0 && out_stride % 2 == 0 && ((uintptr_t)q % 4 == 0) && ((uintptr_t)out % 4 == 0),
                "attention_prefill: q and out must be 4-byte aligned");
#define ZLM_PRE_CASE(H)                                                                                         \
    case H:                                                                                                     \
        return launch_prefill<H>((__nv_bfloat16*)out, out_stride, (const __nv_bfloat16*)q, q_stride,            \
                                 (const __nv_bfloat16*)pool, block_table, table_stride, cu_seqlens, seq_slot,   \
                                 seq_start, R, max_new, nq, nkv, scale, window, sink, opt, st);
    switch (hd) {
        ZLM_PRE_CASE(16) ZLM_PRE_CASE(32) ZLM_PRE_CASE(48) ZLM_PRE_CASE(64) ZLM_PRE_CASE(80) ZLM_PRE_CASE(96)
        ZLM_PRE_CASE(112) ZLM_PRE_CASE(128) ZLM_PRE_CASE(144) ZLM_PRE_CASE(160) ZLM_PRE_CASE(176) ZLM_PRE_CASE(192)
    }
#undef ZLM_PRE_CASE
    ZLM_REQUIRE(false, "attention_prefill: head_dim=%d", hd);
}

// The same with values narrower than keys: the pool's value rows are hd wide but only their first vd columns are
// used (the rest is padding); out's columns from vd on are written as zeros.  Built for a few pairs of widths.
extern "C" int zlm_attention_prefill_vd_supported(int nq, int nkv, int hd, int vd) {
    if (!(nkv > 0 && nq % nkv == 0)) return 0;
    return ((hd == 192 && vd == 128) || (hd == 128 && vd == 64) || (hd == 96 && vd == 64) || (hd == 64 && vd == 32) ||
            (hd == 48 && vd == 32) || (hd == 32 && vd == 16)) ? 1 : 0;
}

extern "C" int zlm_attention_prefill_vd(void* out, int out_stride, const void* q, int q_stride, const void* pool,
                                        const int* block_table, int table_stride, const int* cu_seqlens,
                                        const int* seq_slot, const int* seq_start, int R, int max_new, int nq,
                                        int nkv, int hd, int vd, float scale, int window, int sink, int chunk,
                                        float softcap, const float* sinks, int v_share, int keep, const float* bias,
                                        int bias_n, cudaStream_t st) {
    if (R == 0 || max_new == 0) return ZLM_OK;
    ZLM_REQUIRE(zlm_attention_prefill_vd_supported(nq, nkv, hd, vd),
                "attention_prefill: keys of %d with values of %d columns is not a pair this kernel is built for", hd, vd);
    ZLM_REQUIRE_ATTN_OPTS("attention_prefill");
    const AttnOpts opt{chunk, softcap, sinks, v_share, keep, bias, bias_n};
    ZLM_REQUIRE(q_stride % 2 == 0 && out_stride % 2 == 0 && ((uintptr_t)q % 4 == 0) && ((uintptr_t)out % 4 == 0),
                "attention_prefill: q and out must be 4-byte aligned");
#define ZLM_PRE_VD(H, V)                                                                                           \
    if (hd == H && vd == V)                                                                                        \
        return launch_prefill<H, V>((__nv_bfloat16*)out, out_stride, (const __nv_bfloat16*)q, q_stride,            \
                                    (const __nv_bfloat16*)pool, block_table, table_stride, cu_seqlens, seq_slot,   \
                                    seq_start, R, max_new, nq, nkv, scale, window, sink, opt, st);
    ZLM_PRE_VD(192, 128) ZLM_PRE_VD(128, 64) ZLM_PRE_VD(96, 64) ZLM_PRE_VD(64, 32) ZLM_PRE_VD(48, 32) ZLM_PRE_VD(32, 16)
#undef ZLM_PRE_VD
    ZLM_REQUIRE(false, "attention_prefill: head_dim=%d values=%d", hd, vd);
}

ZLM_TRANSLATION_UNIT(attention_prefill)
