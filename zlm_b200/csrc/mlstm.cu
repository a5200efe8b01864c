// Matrix memory with exponential gates (mLSTM), one matrix S [dim][v_dim] and one vector n [dim] a head:
//   i_t = cap tanh((zi + bi) / cap),  f_t = log sigmoid(cap tanh((zf + bf) / cap))         logarithms of the gates
//   m_t = max(f_t + m_(t-1), i_t)                                                          running maximum, from 0
//   S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T,   n_t likewise with k_t alone
//   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
// q (times q_scale), k, v are columns of a projection in the element type, zi and zf columns of an fp32 buffer.  All that
// follows the projections is fp32 in both element types; sums of many logarithms are kept in 64-bit, so that their
// differences are as good as the token-by-token recurrence's.  A sequence's state is S [slots][H][D][V], n [slots][H][D],
// m [slots][H], read at a step's start and written at its end, zeros in a new slot.
//
// One token a sequence (mlstm_step): a cluster of blocks shares a head's columns, each block updates and reads out its
// strip of S in registers; the heads' unit norm, its weight and the gate sigmoid(g) ride in the same kernel (the sum of
// squares crosses the cluster through distributed shared memory), so that S moves through memory once each way.
//
// Many tokens, in pieces of ML_L tokens side by side.  With b_j the sum of f up to j inside a piece and e_j = i_j - b_j:
//   1. mlstm_piece   what a piece adds to a state, with weights exp(e_l - max e): the product (w k)^T v and the sum of w k
//   2. mlstm_chain   the pieces' states and maxima in order: the state ahead of every piece, and the sequence's new state
//   3. mlstm_out     with M_j = max(m ahead, max_(l <= j) e_l), so that m_j = b_j + M_j:
//                    o_j = (sum_(l <= j) exp(e_l - M_j) (q_j . k_l) v_l + exp(m ahead - M_j) S^T q_j) / ...
#include "common.cuh"
#include <cooperative_groups.h>
namespace cg = cooperative_groups;

#define ML_L 64                  // tokens of a piece
#define ML_THREADS 256
#define ML_COLS 128              // value columns of a block
#define ML_KC 32                 // rows of an operand staged at a time
#define ML_LD 68                 // row of 64 tokens in shared memory: 16-byte accesses of a column by neighbouring lanes meet no bank twice

struct MlstmGates {
    const float* z;              // [T][stride]: zi of head h in column i_off + h, zf in f_off + h
    int stride, i_off, f_off;
    VecW bi, bf;
    float cap;
};
__device__ __forceinline__ float ml_cap(float x, float cap) { return cap > 0.f ? cap * tanhf(x / cap) : x; }
// (log input gate, log forget gate) of a token's head
__device__ __forceinline__ float2 ml_gates(const MlstmGates& g, size_t row, int h) {
    const float* z = g.z + row * g.stride;
    if (!ZLM_CHK(z + g.i_off + h, 4) || !ZLM_CHK(z + g.f_off + h, 4)) return make_float2(0.f, 0.f);
    const float x = ml_cap(z[g.f_off + h] + (g.bf.p ? g.bf[h] : 0.f), g.cap);
    return make_float2(ml_cap(z[g.i_off + h] + (g.bi.p ? g.bi[h] : 0.f), g.cap), fminf(x, 0.f) - log1pf(expf(-fabsf(x))));
}
__device__ __forceinline__ float ml_denominator(float nq, float m) { return fmaxf(fabsf(nq), expf(-m)) + 1e-6f; }

template <int VEC> struct MlVec { float v[VEC]; };
template <int VEC> __device__ __forceinline__ MlVec<VEC> ml_load(const float* p) {
    MlVec<VEC> r;
    if (VEC == 4) {
        const float4 a = *(const float4*)p;
        r.v[0] = a.x; r.v[VEC > 1 ? 1 : 0] = a.y; r.v[VEC > 2 ? 2 : 0] = a.z; r.v[VEC > 3 ? 3 : 0] = a.w;
        return r;
    }
    r.v[0] = p[0];
    return r;
}
template <int VEC> __device__ __forceinline__ void ml_store(float* p, const MlVec<VEC>& r) {
    if (VEC == 4) *(float4*)p = make_float4(r.v[0], r.v[VEC > 1 ? 1 : 0], r.v[VEC > 2 ? 2 : 0], r.v[VEC > 3 ? 3 : 0]);
    else p[0] = r.v[0];
}

// ---------------------------------------------------------------------------- one token a sequence
// grid (R * cluster, H), clusters along x; a block owns the columns [rank * VC, ...) of one head of one sequence.  A thread
// owns VEC neighbouring columns of every RG-th row.
#define ML_AHEAD 4
template <typename TA, typename TO, int VEC>
__global__ void __launch_bounds__(ML_THREADS, 4)
mlstm_step_kernel(TO* __restrict__ out, int out_stride, const TA* __restrict__ proj, int stride, int q_off, int k_off, int v_off,
                  int g_off, MlstmGates gates, float* __restrict__ S, float* __restrict__ nvec, float* __restrict__ mmax,
                  const int* __restrict__ seq_slot, const int* __restrict__ cu_seqlens, int H, int D, int V, int VC, float q_scale,
                  VecW w_norm, float eps) {
    cg::cluster_group cluster = cg::this_cluster();
    extern __shared__ __align__(16) float ml_smem[];       // q [D], k [D], new n [D], sums [rows][VC], o [VC]
    __shared__ float red[32];
    __shared__ float squares;
    const int NS = cluster.num_blocks(), rank = cluster.block_rank();
    const int r = blockIdx.x / NS, h = blockIdx.y, tid = threadIdx.x;
    const int CG = VC / VEC, RG = ML_THREADS / CG;
    const int rg = tid / CG, cc = (tid - rg * CG) * VEC;
    const bool folds = 32 % CG == 0 && RG * CG == ML_THREADS;      // a warp holds whole rows: their sums meet in shuffles first
    const int rows = folds ? ML_THREADS / 32 : RG;
    const int c0 = rank * VC, ncol = max(0, min(VC, V - c0));
    const bool live = rg < RG && cc < ncol;
    float* sq = ml_smem;
    float* sk = sq + D;
    float* sn = sk + D;
    float* sums = sn + D;
    float* so = sums + rows * VC;
    const bool ok = ZLM_CHK(seq_slot + r, 4) && ZLM_CHK(cu_seqlens + r, 4);      // (block-uniform; the cluster's barriers below are met either way)
    const int slot = ok ? seq_slot[r] : 0;
    const size_t t = ok ? cu_seqlens[r] : 0;
    const size_t sh = (size_t)slot * H + h;
    float* sp = S + (sh * D) * V + c0 + cc;
    // the state is from earlier steps: its first rows are on the way before the wait for the projection
    MlVec<VEC> s[ML_AHEAD];
    auto load_rows = [&](int d0) {
#pragma unroll
        for (int j = 0; j < ML_AHEAD; ++j) {
            const int d = d0 + j * RG;
            if (live && d < D && ZLM_CHK(sp + (size_t)d * V, VEC * 4)) s[j] = ml_load<VEC>(sp + (size_t)d * V);
            else memset(&s[j], 0, sizeof(s[j]));
        }
    };
    load_rows(rg);
    pdl_trigger();
    pdl_wait();
    const TA* row = proj + t * stride;
    for (int d = tid; d < D; d += ML_THREADS) {
        sq[d] = ZLM_CHK(row + q_off + h * D + d, sizeof(TA)) ? to_f32(row[q_off + h * D + d]) * q_scale : 0.f;
        sk[d] = ZLM_CHK(row + k_off + h * D + d, sizeof(TA)) ? to_f32(row[k_off + h * D + d]) : 0.f;
    }
    const float2 lg = ml_gates(gates, t, h);
    const float m_old = ZLM_CHK(mmax + sh, 4) ? mmax[sh] : 0.f;
    const float m = fmaxf(lg.y + m_old, lg.x);
    const float keep = expf(lg.y + m_old - m), take = expf(lg.x - m);
    float nq = 0.f;
    for (int d = tid; d < D; d += ML_THREADS) {             // (a thread's own q and k: no barrier in between)
        const float* np = nvec + sh * D + d;
        sn[d] = fmaf(keep, ZLM_CHK(np, 4) ? *np : 0.f, take * sk[d]);
        nq = fmaf(sn[d], sq[d], nq);
    }
    float v[VEC], acc[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        const TA* vp = row + v_off + (size_t)h * V + c0 + cc + e;
        v[e] = (live && ZLM_CHK(vp, sizeof(TA))) ? to_f32(*vp) * take : 0.f;
        acc[e] = 0.f;
    }
    nq = block_sum(nq, red);                                // (its barriers also publish q, k and n)
    if (live) {
        for (int d0 = rg; d0 < D; d0 += ML_AHEAD * RG) {
#pragma unroll
            for (int j = 0; j < ML_AHEAD; ++j) {
                const int d = d0 + j * RG;
                if (d >= D) break;
                const float kd = sk[d], qd = sq[d];
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    s[j].v[e] = fmaf(keep, s[j].v[e], kd * v[e]);
                    acc[e] = fmaf(s[j].v[e], qd, acc[e]);
                }
                if (ZLM_CHK(sp + (size_t)d * V, VEC * 4)) ml_store<VEC>(sp + (size_t)d * V, s[j]);
            }
            load_rows(d0 + ML_AHEAD * RG);
        }
    }
    if (folds) {
#pragma unroll
        for (int e = 0; e < VEC; ++e)
            for (int x = CG; x < 32; x <<= 1) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], x);
    }
    if (live && (!folds || (tid & 31) < CG)) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) sums[(folds ? tid >> 5 : rg) * VC + cc + e] = acc[e];
    }
    __syncthreads();
    const float den = ml_denominator(nq, m);
    float ss = 0.f;
    for (int c = tid; c < ncol; c += ML_THREADS) {
        float o = 0.f;
        for (int x = 0; x < rows; ++x) o += sums[x * VC + c];
        o /= den;
        so[c] = o;
        ss = fmaf(o, o, ss);
    }
    ss = block_sum(ss, red);
    if (tid == 0) squares = ss;
    cluster.sync();
    // every block of the cluster has read the old n and m; one writes the new ones
    if (rank == 0 && ok) {
        for (int d = tid; d < D; d += ML_THREADS)
            if (ZLM_CHK(nvec + sh * D + d, 4)) nvec[sh * D + d] = sn[d];
        if (tid == 0 && ZLM_CHK(mmax + sh, 4)) mmax[sh] = m;
    }
    float total = 0.f;
    for (int k = 0; k < NS; ++k) total += *cluster.map_shared_rank(&squares, k);
    const float inv = 1.0f / sqrtf(total / (float)V + eps);
    for (int c = tid; c < ncol; c += ML_THREADS) {
        const int hv = h * V + c0 + c;
        const TA* gp = row + g_off + hv;
        TO* op = out + t * out_stride + hv;
        if (ok && ZLM_CHK(gp, sizeof(TA)) && ZLM_CHK(op, sizeof(TO)))
            *op = from_f32<TO>(so[c] * inv * w_norm[hv] / (1.0f + expf(-to_f32(*gp))));
    }
    cluster.sync();                  // no block leaves while another may still read its sum
}

// ---------------------------------------------------------------------------- pieces of many tokens
// What one warp works out about a piece: b (sums of log forget gates, inclusive) and e = i - b per token, in 64-bit, into
// shared memory [ML_L] each; tokens from n on have f = 0 and e = -infinity.  Returns (b of the whole piece, the largest e).
__device__ __forceinline__ double2 ml_piece_gates(const MlstmGates& gates, size_t row0, int n, int h, double* sb, double* se) {
    const int lane = threadIdx.x & 31;
    float2 g[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) g[x] = 2 * lane + x < n ? ml_gates(gates, row0 + 2 * lane + x, h) : make_float2(-INFINITY, 0.f);
    const double own = (double)g[0].y + (double)g[1].y;
    double sum = own;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += up;
    }
    const double b0 = sum - (double)g[1].y, b1 = sum;
    const double e0 = (double)g[0].x - b0, e1 = (double)g[1].x - b1;
    sb[2 * lane] = b0; sb[2 * lane + 1] = b1;
    se[2 * lane] = e0; se[2 * lane + 1] = e1;
    double mx = fmax(e0, e1);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmax(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    return make_double2(__shfl_sync(0xffffffffu, sum, 31), mx);
}

// eight neighbouring elements of a row, zeros where `ok` is false or beyond `left` of them
template <typename TA>
__device__ __forceinline__ void ml_load8(const TA* p, int left, bool ok, bool vec, float* f) {
    if (ok && vec && left >= 8 && ZLM_CHK(p, 8 * sizeof(TA))) {
        if (sizeof(TA) == 2) {
            const uint4 u = *(const uint4*)p;
            f[0] = __uint_as_float(u.x << 16); f[1] = __uint_as_float(u.x & 0xffff0000u);
            f[2] = __uint_as_float(u.y << 16); f[3] = __uint_as_float(u.y & 0xffff0000u);
            f[4] = __uint_as_float(u.z << 16); f[5] = __uint_as_float(u.z & 0xffff0000u);
            f[6] = __uint_as_float(u.w << 16); f[7] = __uint_as_float(u.w & 0xffff0000u);
        } else {
            const float4 a = *(const float4*)p, b = *(const float4*)((const float*)p + 4);
            f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
        }
        return;
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = (ok && e < left && ZLM_CHK(p + e, sizeof(TA))) ? to_f32(p[e]) : 0.f;
}

// the same in two steps: fetched as stored, widened later
template <typename TA> struct MlRaw8 { float v[8]; };
template <> struct MlRaw8<__nv_bfloat16> { uint4 v; };
template <typename TA> __device__ __forceinline__ MlRaw8<TA> ml_fetch8(const TA* p, int left, bool ok, bool vec) {
    MlRaw8<TA> r;
    if constexpr (sizeof(TA) == 2) {
        if (ok && vec && left >= 8 && ZLM_CHK(p, 16)) {
            r.v = *(const uint4*)p;
        } else {
            unsigned short h[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) h[e] = (ok && e < left && ZLM_CHK(p + e, 2)) ? *(const unsigned short*)(p + e) : (unsigned short)0;
            r.v = make_uint4(h[0] | (unsigned)h[1] << 16, h[2] | (unsigned)h[3] << 16, h[4] | (unsigned)h[5] << 16, h[6] | (unsigned)h[7] << 16);
        }
    } else {
        ml_load8<TA>(p, left, ok, vec, r.v);
    }
    return r;
}
__device__ __forceinline__ void ml_widen8(const MlRaw8<float>& r, float* f) {
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = r.v[e];
}
__device__ __forceinline__ void ml_widen8(const MlRaw8<__nv_bfloat16>& r, float* f) {
    f[0] = __uint_as_float(r.v.x << 16); f[1] = __uint_as_float(r.v.x & 0xffff0000u);
    f[2] = __uint_as_float(r.v.y << 16); f[3] = __uint_as_float(r.v.y & 0xffff0000u);
    f[4] = __uint_as_float(r.v.z << 16); f[5] = __uint_as_float(r.v.z & 0xffff0000u);
    f[6] = __uint_as_float(r.v.w << 16); f[7] = __uint_as_float(r.v.w & 0xffff0000u);
}

// acc[8][4] += X^T Y over `kn` staged rows: X [kn][ML_LD], the warp's eight columns; Y [kn][ML_COLS], the lane's four
__device__ __forceinline__ void ml_multiply(float (&acc)[8][4], const float* X, const float* Y, int kn, int warp, int lane) {
#pragma unroll 4
    for (int k = 0; k < kn; ++k) {
        const float4 xa = *(const float4*)(X + k * ML_LD + warp * 8), xb = *(const float4*)(X + k * ML_LD + warp * 8 + 4);
        const float4 y = *(const float4*)(Y + k * ML_COLS + lane * 4);
        const float x[8] = {xa.x, xa.y, xa.z, xa.w, xb.x, xb.y, xb.z, xb.w};
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            acc[i][0] = fmaf(x[i], y.x, acc[i][0]);
            acc[i][1] = fmaf(x[i], y.y, acc[i][1]);
            acc[i][2] = fmaf(x[i], y.z, acc[i][2]);
            acc[i][3] = fmaf(x[i], y.w, acc[i][3]);
        }
    }
}

struct MlPiece {
    int r, p, h, slot, row0, n;          // sequence, piece, head, slot; the piece's first row and tokens
    size_t at;                           // (piece, head) in the scratch arrays
};
__device__ __forceinline__ bool ml_piece(MlPiece& x, int unit, int H, int maxp, const int* seq_slot, const int* cu_seqlens) {
    x.h = unit % H;
    const int rp = unit / H;
    x.r = rp / maxp;
    x.p = rp % maxp;
    if (!ZLM_CHK(seq_slot + x.r, 4) || !ZLM_CHK(cu_seqlens + x.r, 8)) return false;
    x.slot = seq_slot[x.r];
    x.row0 = cu_seqlens[x.r] + x.p * ML_L;
    x.n = min(ML_L, cu_seqlens[x.r + 1] - x.row0);
    x.at = (size_t)unit;
    return x.n > 0;
}

// grid (R * maxp * H, ceil(D / 64), ceil(V / 128))
template <typename TA>
__global__ void __launch_bounds__(ML_THREADS)
mlstm_piece_kernel(float* __restrict__ part, float* __restrict__ part_n, float2* __restrict__ part_m, const TA* __restrict__ proj,
                   int stride, int k_off, int v_off, MlstmGates gates, const int* __restrict__ seq_slot,
                   const int* __restrict__ cu_seqlens, int H, int D, int V, int maxp, int vec) {
    extern __shared__ __align__(16) float ml_smem[];
    float* X = ml_smem;                          // [ML_L][ML_LD]: w_l k_l
    float* Y = X + ML_L * ML_LD;                   // [ML_L][ML_COLS]: v_l
    __shared__ double sb[ML_L], se[ML_L], top;
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int d0 = blockIdx.y * 64, c0 = blockIdx.z * ML_COLS;
    MlPiece pc;
    pdl_wait();
    if (!ml_piece(pc, blockIdx.x, H, maxp, seq_slot, cu_seqlens)) return;         // block-uniform
    // the keys and values are on their way while the gates are worked out
    float fk[ML_L * 8 / ML_THREADS][8];
#pragma unroll
    for (int y = 0; y < ML_L * 8 / ML_THREADS; ++y) {
        const int x = tid + y * ML_THREADS, l = x / 8, d = (x % 8) * 8;
        ml_load8<TA>(proj + (size_t)(pc.row0 + l) * stride + k_off + (size_t)pc.h * D + d0 + d, D - d0 - d, l < pc.n, vec, fk[y]);
    }
    if (warp == 0) {
        const double2 g = ml_piece_gates(gates, pc.row0, pc.n, pc.h, sb, se);
        if (lane == 0) {
            top = g.y;
            if (blockIdx.y == 0 && blockIdx.z == 0 && ZLM_CHK(part_m + pc.at, 8)) part_m[pc.at] = make_float2((float)g.x, (float)(g.x + g.y));
        }
    }
    for (int x = tid; x < ML_L * (ML_COLS / 8); x += ML_THREADS) {
        const int l = x / (ML_COLS / 8), c = (x % (ML_COLS / 8)) * 8;
        float f[8];
        ml_load8<TA>(proj + (size_t)(pc.row0 + l) * stride + v_off + (size_t)pc.h * V + c0 + c, V - c0 - c, l < pc.n, vec, f);
        *(float4*)(Y + l * ML_COLS + c) = make_float4(f[0], f[1], f[2], f[3]);
        *(float4*)(Y + l * ML_COLS + c + 4) = make_float4(f[4], f[5], f[6], f[7]);
    }
    __syncthreads();
#pragma unroll
    for (int y = 0; y < ML_L * 8 / ML_THREADS; ++y) {
        const int x = tid + y * ML_THREADS, l = x / 8, d = (x % 8) * 8;
        const float* f = fk[y];
        const float w = l < pc.n ? expf((float)(se[l] - top)) : 0.f;
        *(float4*)(X + l * ML_LD + d) = make_float4(f[0] * w, f[1] * w, f[2] * w, f[3] * w);
        *(float4*)(X + l * ML_LD + d + 4) = make_float4(f[4] * w, f[5] * w, f[6] * w, f[7] * w);
    }
    __syncthreads();
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    ml_multiply(acc, X, Y, pc.n, warp, lane);
    const int c = c0 + lane * 4;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int d = d0 + warp * 8 + i;
        if (d >= D) continue;
        float* dst = part + (pc.at * D + d) * V + c;
        if ((V & 3) == 0 && c < V && ZLM_CHK(dst, 16)) {
            *(float4*)dst = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (c + j < V && ZLM_CHK(dst + j, 4)) dst[j] = acc[i][j];
        }
    }
    if (blockIdx.z == 0 && tid < 64 && d0 + tid < D) {
        float s = 0.f;
        for (int l = 0; l < pc.n; ++l) s += X[l * ML_LD + tid];
        float* dst = part_n + pc.at * D + d0 + tid;
        if (ZLM_CHK(dst, 4)) *dst = s;
    }
}

// The pieces' states in order: part and part_n become the state ahead of the piece, `ahead` the maxima ahead of it and
// after it; S and n of the sequence are left.  A thread owns VEC neighbouring numbers of S; the blocks with
// blockIdx.y == 0 also chain n.  grid (R * H, ceil(D * V / (128 VEC)))
#define ML_CHAIN 8
template <int VEC>
__global__ void __launch_bounds__(128)
mlstm_chain_kernel(float* __restrict__ part, float* __restrict__ part_n, const float2* __restrict__ part_m, float2* __restrict__ ahead,
                   float* __restrict__ S, float* __restrict__ nvec, const float* __restrict__ mmax, const int* __restrict__ seq_slot,
                   const int* __restrict__ cu_seqlens, int H, int D, int V, int maxp) {
    pdl_launch_dependents();
    const int r = blockIdx.x / H, h = blockIdx.x % H, tid = threadIdx.x;
    pdl_wait();
    if (!ZLM_CHK(seq_slot + r, 4) || !ZLM_CHK(cu_seqlens + r, 8)) return;
    const int slot = seq_slot[r], np = (cu_seqlens[r + 1] - cu_seqlens[r] + ML_L - 1) / ML_L;
    const size_t DV = (size_t)D * V, sh = (size_t)slot * H + h, e = ((size_t)blockIdx.y * 128 + tid) * VEC;
    const bool live = e < DV && ZLM_CHK(S + sh * DV + e, VEC * 4);
    MlVec<VEC> s;
    memset(&s, 0, sizeof(s));
    if (live) s = ml_load<VEC>(S + sh * DV + e);
    float m = ZLM_CHK(mmax + sh, 4) ? mmax[sh] : 0.f;
    const size_t at0 = (size_t)r * maxp * H + h;
    for (int p0 = 0; p0 < np; p0 += ML_CHAIN) {
        const int cnt = min(ML_CHAIN, np - p0);
        MlVec<VEC> a[ML_CHAIN];
#pragma unroll
        for (int j = 0; j < ML_CHAIN; ++j) {
            const float* src = part + (at0 + (size_t)(p0 + j) * H) * DV + e;
            if (live && j < cnt && ZLM_CHK(src, VEC * 4)) a[j] = ml_load<VEC>(src);
            else memset(&a[j], 0, sizeof(a[j]));
        }
        // (factor of the state ahead, factor of the piece's own part): every thread works them out for itself
        float2 coef[ML_CHAIN];
#pragma unroll
        for (int j = 0; j < ML_CHAIN; ++j) {
            const float2* src = part_m + at0 + (size_t)(p0 + j) * H;
            coef[j] = (j < cnt && ZLM_CHK(src, 8)) ? *src : make_float2(0.f, 0.f);
        }
#pragma unroll
        for (int j = 0; j < ML_CHAIN; ++j) {
            if (j >= cnt) break;
            const float2 g = coef[j];
            const float next = fmaxf(g.x + m, g.y);
            coef[j] = make_float2(expf(g.x + m - next), expf(g.y - next));
            float2* dst = ahead + at0 + (size_t)(p0 + j) * H;
            if (blockIdx.y == 0 && tid == 0 && ZLM_CHK(dst, 8)) *dst = make_float2(m, next);
            m = next;
        }
#pragma unroll
        for (int j = 0; j < ML_CHAIN; ++j) {
            if (j >= cnt) break;
            float* dst = part + (at0 + (size_t)(p0 + j) * H) * DV + e;
            if (live && ZLM_CHK(dst, VEC * 4)) ml_store<VEC>(dst, s);
            const float2 c = coef[j];
#pragma unroll
            for (int x = 0; x < VEC; ++x) s.v[x] = fmaf(c.x, s.v[x], c.y * a[j].v[x]);
        }
        if (blockIdx.y == 0) {
            for (int d = tid; d < D; d += 128) {
                float* np_ = nvec + sh * D + d;
                if (!ZLM_CHK(np_, 4)) continue;
                float n = *np_, own[ML_CHAIN];
#pragma unroll
                for (int j = 0; j < ML_CHAIN; ++j) {
                    const float* q = part_n + (at0 + (size_t)(p0 + j) * H) * D + d;
                    own[j] = (j < cnt && ZLM_CHK(q, 4)) ? *q : 0.f;
                }
#pragma unroll
                for (int j = 0; j < ML_CHAIN; ++j) {
                    if (j >= cnt) break;
                    float* q = part_n + (at0 + (size_t)(p0 + j) * H) * D + d;
                    if (ZLM_CHK(q, 4)) *q = n;
                    n = fmaf(coef[j].x, n, coef[j].y * own[j]);
                }
                *np_ = n;
            }
        }
    }
    if (live) ml_store<VEC>(S + sh * DV + e, s);
}

// grid (R * maxp * H, ceil(V / 128))
template <typename TA>
__global__ void __launch_bounds__(ML_THREADS, 2)
mlstm_out_kernel(float* __restrict__ o, const TA* __restrict__ proj, int stride, int q_off, int k_off, int v_off, MlstmGates gates,
                 const float* __restrict__ part, const float* __restrict__ part_n, const float2* __restrict__ ahead,
                 float* __restrict__ mmax, const int* __restrict__ seq_slot, const int* __restrict__ cu_seqlens, int H, int D, int V,
                 int maxp, float q_scale, int vec) {
    extern __shared__ __align__(16) float ml_smem[];
    float* Q = ml_smem;                          // [ML_KC][ML_LD]: 32 coordinates of the tokens' queries
    float* K = Q + ML_KC * ML_LD;                // [ML_KC][ML_LD]: and of their keys
    float* P = K + ML_KC * ML_LD;                // [ML_L keys][ML_LD: tokens]
    float* Y = P + ML_L * ML_LD;                 // [2][ML_KC][ML_COLS]: rows of the state ahead, then values
    __shared__ double sb[ML_L], se[ML_L], sm[ML_L];
    __shared__ float snv[ML_KC];
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int c0 = blockIdx.y * ML_COLS;
    MlPiece pc;
    pdl_wait();
    if (!ml_piece(pc, blockIdx.x, H, maxp, seq_slot, cu_seqlens)) return;         // block-uniform
    if (!ZLM_CHK(ahead + pc.at, 8)) return;
    const float2 ma = ahead[pc.at];
    // a chunk of 32 coordinates: queries and keys through registers (they are turned round on the way), rows of the state
    // straight into shared memory; the next chunk is on its way while this one's products run
    MlRaw8<TA> rq, rk;
    const int ql = tid & 63, qd = (tid >> 6) * 8;
    auto fetch = [&](int d0, int buf) {
        const TA* row = proj + (size_t)(pc.row0 + ql) * stride + (size_t)pc.h * D + d0 + qd;
        rq = ml_fetch8<TA>(row + q_off, D - d0 - qd, ql < pc.n, vec);
        rk = ml_fetch8<TA>(row + k_off, D - d0 - qd, ql < pc.n, vec);
        for (int x = tid; x < ML_KC * (ML_COLS / 4); x += ML_THREADS) {
            const int d = x / (ML_COLS / 4), c = (x % (ML_COLS / 4)) * 4;
            const float* src = part + (pc.at * D + d0 + d) * V + c0 + c;
            float* dst = Y + (size_t)buf * ML_KC * ML_COLS + d * ML_COLS + c;
            if (d0 + d < D && (V & 3) == 0 && c0 + c < V && ZLM_CHK(src, 16)) {
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src));
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) dst[e] = (d0 + d < D && c0 + c + e < V && ZLM_CHK(src + e, 4)) ? src[e] : 0.f;
            }
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
    fetch(0, 0);
    if (warp == 0) {
        ml_piece_gates(gates, pc.row0, pc.n, pc.h, sb, se);
        __syncwarp();
        // M: the running maximum of e and of the maximum ahead
        const double e0 = se[2 * lane], e1 = fmax(e0, se[2 * lane + 1]);
        double mx = e1;
#pragma unroll
        for (int x = 1; x < 32; x <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, mx, x);
            if (lane >= x) mx = fmax(mx, up);
        }
        double before = __shfl_up_sync(0xffffffffu, mx, 1);
        before = lane ? fmax(before, (double)ma.x) : (double)ma.x;
        sm[2 * lane] = fmax(before, e0);
        sm[2 * lane + 1] = fmax(before, e1);
        // the sequence's new maximum, from its last piece
        if (lane == 0 && blockIdx.y == 0 && (pc.p + 1) * ML_L >= cu_seqlens[pc.r + 1] - cu_seqlens[pc.r]) {
            float* dst = mmax + (size_t)pc.slot * H + pc.h;
            if (ZLM_CHK(dst, 4)) *dst = ma.y;
        }
    }
    float acc[8][4], p[8][2], nq[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        p[i][0] = p[i][1] = nq[i] = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    }
    for (int d0 = 0, buf = 0; d0 < D; d0 += ML_KC, buf ^= 1) {
        __syncthreads();                         // (the products of the chunk before are done)
        {
            float fq[8], fk[8];
            ml_widen8(rq, fq);
            ml_widen8(rk, fk);
#pragma unroll
            for (int x = 0; x < 8; ++x) {
                Q[(qd + x) * ML_LD + ql] = fq[x] * q_scale;
                K[(qd + x) * ML_LD + ql] = fk[x];
            }
        }
        if (tid < ML_KC) snv[tid] = (d0 + tid < D && ZLM_CHK(part_n + pc.at * D + d0 + tid, 4)) ? part_n[pc.at * D + d0 + tid] : 0.f;
        if (d0 + ML_KC < D) {
            fetch(d0 + ML_KC, buf ^ 1);
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();
        const float* Yb = Y + (size_t)buf * ML_KC * ML_COLS;
        const int kn = min(ML_KC, D - d0);
#pragma unroll 4
        for (int k = 0; k < kn; ++k) {
            const float4 qa = *(const float4*)(Q + k * ML_LD + warp * 8), qb = *(const float4*)(Q + k * ML_LD + warp * 8 + 4);
            const float4 y = *(const float4*)(Yb + k * ML_COLS + lane * 4);
            const float k0 = K[k * ML_LD + lane], k1 = K[k * ML_LD + 32 + lane];            // (a lane's keys: lane and 32 + lane)
            const float q[8] = {qa.x, qa.y, qa.z, qa.w, qb.x, qb.y, qb.z, qb.w};
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                acc[i][0] = fmaf(q[i], y.x, acc[i][0]);
                acc[i][1] = fmaf(q[i], y.y, acc[i][1]);
                acc[i][2] = fmaf(q[i], y.z, acc[i][2]);
                acc[i][3] = fmaf(q[i], y.w, acc[i][3]);
                p[i][0] = fmaf(q[i], k0, p[i][0]);
                p[i][1] = fmaf(q[i], k1, p[i][1]);
            }
        }
        // n ahead . q: a lane takes one coordinate of the warp's eight tokens
        const float nv = snv[lane];
#pragma unroll
        for (int i = 0; i < 8; i += 4) {
            const float4 q4 = *(const float4*)(Q + lane * ML_LD + warp * 8 + i);
            nq[i] = fmaf(nv, q4.x, nq[i]);
            nq[i + 1] = fmaf(nv, q4.y, nq[i + 1]);
            nq[i + 2] = fmaf(nv, q4.z, nq[i + 2]);
            nq[i + 3] = fmaf(nv, q4.w, nq[i + 3]);
        }
    }
    // the weights of the piece's own keys, and the denominators
    float den[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int j = warp * 8 + i;
        const double M = sm[j];
        const float c = expf((float)((double)ma.x - M));
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int l = lane + 32 * x;
            p[i][x] = (l <= j && l < pc.n) ? p[i][x] * expf((float)(se[l] - M)) : 0.f;
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) acc[i][x] *= c;
        den[i] = ml_denominator(warp_sum(fmaf(c, nq[i], p[i][0] + p[i][1])), (float)(sb[j] + M));
    }
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        float* dst = P + (lane + 32 * x) * ML_LD + warp * 8;
        *(float4*)dst = make_float4(p[0][x], p[1][x], p[2][x], p[3][x]);
        *(float4*)(dst + 4) = make_float4(p[4][x], p[5][x], p[6][x], p[7][x]);
    }
    for (int l0 = 0; l0 < pc.n; l0 += ML_KC) {
        __syncthreads();
        for (int x = tid; x < ML_KC * (ML_COLS / 8); x += ML_THREADS) {
            const int l = x / (ML_COLS / 8), c = (x % (ML_COLS / 8)) * 8;
            float f[8];
            ml_load8<TA>(proj + (size_t)(pc.row0 + l0 + l) * stride + v_off + (size_t)pc.h * V + c0 + c, V - c0 - c, l0 + l < pc.n, vec, f);
            *(float4*)(Y + l * ML_COLS + c) = make_float4(f[0], f[1], f[2], f[3]);
            *(float4*)(Y + l * ML_COLS + c + 4) = make_float4(f[4], f[5], f[6], f[7]);
        }
        __syncthreads();
        // (a warp's tokens see no key after its last one)
        ml_multiply(acc, P + l0 * ML_LD, Y, max(0, min(min(ML_KC, pc.n - l0), warp * 8 + 8 - l0)), warp, lane);
    }
    const int c = c0 + lane * 4;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int j = warp * 8 + i;
        if (j >= pc.n) continue;
        const float inv = 1.0f / den[i];
        float* dst = o + ((size_t)(pc.row0 + j) * H + pc.h) * V + c;
        if ((V & 3) == 0 && c < V && ZLM_CHK(dst, 16)) {
            *(float4*)dst = make_float4(acc[i][0] * inv, acc[i][1] * inv, acc[i][2] * inv, acc[i][3] * inv);
        } else {
#pragma unroll
            for (int x = 0; x < 4; ++x)
                if (c + x < V && ZLM_CHK(dst + x, 4)) dst[x] = acc[i][x] * inv;
        }
    }
}

// ---------------------------------------------------------------------------- entry points
static int mlstm_check(const float* z, int H, int D, int V, int R) {
    ZLM_REQUIRE(H > 0 && H <= 65535 && D > 0 && D <= 4096 && V > 0 && R > 0 && z, "mlstm: %d heads of %d key and %d value columns, %d sequences", H, D, V, R);
    return ZLM_OK;
}

template <typename TA, typename TO, int VEC>
static int launch_step(int R, int H, int NS, size_t smem, cudaStream_t st, TO* out, int out_stride, const TA* proj, int stride,
                       int q_off, int k_off, int v_off, int g_off, MlstmGates gates, float* S, float* n, float* m,
                       const int* seq_slot, const int* cu_seqlens, int D, int V, int VC, float q_scale, VecW w_norm, float eps) {
    auto kern = mlstm_step_kernel<TA, TO, VEC>;
    static bool attr_set_dev[64] = {};
    bool& attr_set = attr_set_dev[zlm_device_index()];
    if (smem > 40 * 1024 && !attr_set) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (e != cudaSuccess) {
            zlm_set_error("mlstm_step: cannot reserve shared memory: %s", cudaGetErrorString(e));
            return ZLM_ERR_CUDA;
        }
        attr_set = true;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(R * NS, H);
    cfg.blockDim = dim3(ML_THREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = NS;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = zlm_pdl_enabled() ? 2 : 1;
    zlm_count_launch();
    cudaLaunchKernelEx(&cfg, kern, out, out_stride, proj, stride, q_off, k_off, v_off, g_off, gates, S, n, m, seq_slot, cu_seqlens, H,
                       D, V, VC, q_scale, w_norm, eps);
    return zlm_check_launch("mlstm_step");
}

// blocks of a cluster and the columns of each: strips of about 32 columns, at most eight of them
static int mlstm_strips(int V, int vec, int* cols) {
    int ns = (V + 31) / 32;
    if (ns > 8) ns = 8;
    int vc = (V + ns - 1) / ns;
    vc = (vc + vec - 1) / vec * vec;
    *cols = vc;
    return (V + vc - 1) / vc;
}

// One token a sequence (row cu_seqlens[r] of the step).  proj [T][stride] in `dtype`: q, k from q_off, k_off on (H heads of
// D), v and the output gate's logits from v_off, g_off on (H heads of V); z [T][z_stride] fp32: zi and zf of the heads from
// i_off, f_off on, without the biases bi, bf [H] (null: none).  out [T][out_stride] in out_dtype receives
// o / rms(o of its head) * w_norm[h * V + c] * sigmoid(g).
extern "C" int zlm_mlstm_step(void* out, int out_stride, int out_dtype, const void* proj, int stride, int dtype, int q_off, int k_off,
                              int v_off, int g_off, const float* z, int z_stride, int i_off, int f_off, const void* bi, const void* bf,
                              int b_dtype, float cap, float* S, float* n, float* m, const int* seq_slot, const int* cu_seqlens, int R,
                              int H, int D, int V, float q_scale, const void* w_norm, int w_dtype, float eps, cudaStream_t st) {
    if (R == 0) return ZLM_OK;
    if (int rc = mlstm_check(z, H, D, V, R)) return rc;
    const MlstmGates gates{z, z_stride, i_off, f_off, VecW{bi, b_dtype}, VecW{bf, b_dtype}, cap};
    const int vec = V % 4 == 0 && (uintptr_t)S % 16 == 0 ? 4 : 1;
    int VC;
    const int NS = mlstm_strips(V, vec, &VC);
    ZLM_REQUIRE(VC / vec <= ML_THREADS && (long long)R * NS <= 2147483647LL, "mlstm_step: heads of %d value columns", V);
    const int CG = VC / vec, RG = ML_THREADS / CG;
    const int rows = 32 % CG == 0 && RG * CG == ML_THREADS ? ML_THREADS / 32 : RG;
    const size_t smem = (size_t)(3 * D + rows * VC + VC) * sizeof(float);
    ZLM_REQUIRE(smem <= 200 * 1024, "mlstm_step: %zu bytes a block", smem);
    const VecW wn{w_norm, w_dtype};
#define ZLM_ML_STEP(TA, TO)                                                                                                     \
    return vec == 4 ? launch_step<TA, TO, 4>(R, H, NS, smem, st, (TO*)out, out_stride, (const TA*)proj, stride, q_off, k_off, v_off, \
                                             g_off, gates, S, n, m, seq_slot, cu_seqlens, D, V, VC, q_scale, wn, eps)            \
                    : launch_step<TA, TO, 1>(R, H, NS, smem, st, (TO*)out, out_stride, (const TA*)proj, stride, q_off, k_off, v_off, \
                                             g_off, gates, S, n, m, seq_slot, cu_seqlens, D, V, VC, q_scale, wn, eps)
    if (dtype == ZLM_DTYPE_F32 && out_dtype == ZLM_DTYPE_F32) { ZLM_ML_STEP(float, float); }
    if (dtype == ZLM_DTYPE_F32 && out_dtype == ZLM_DTYPE_BF16) { ZLM_ML_STEP(float, __nv_bfloat16); }
    if (dtype == ZLM_DTYPE_BF16 && out_dtype == ZLM_DTYPE_BF16) { ZLM_ML_STEP(__nv_bfloat16, __nv_bfloat16); }
#undef ZLM_ML_STEP
    ZLM_REQUIRE(false, "mlstm_step: unsupported dtypes %d, %d", dtype, out_dtype);
}

// floats of scratch that zlm_mlstm wants
extern "C" long long zlm_mlstm_scratch(int R, int H, int D, int V, int max_new) {
    const long long maxp = (max_new + ML_L - 1) / ML_L;
    return (long long)R * maxp * H * ((long long)D * V + D + 4);
}

// Any number of tokens a sequence: as zlm_mlstm_step, without the norm and the gate; o [T][H * V] fp32.
extern "C" int zlm_mlstm(float* o, const void* proj, int stride, int dtype, int q_off, int k_off, int v_off, const float* z,
                         int z_stride, int i_off, int f_off, const void* bi, const void* bf, int b_dtype, float cap, float* S, float* n,
                         float* m, const int* seq_slot, const int* cu_seqlens, int T, int R, int H, int D, int V, float q_scale,
                         int max_new, float* scratch, cudaStream_t st) {
    if (T == 0) return ZLM_OK;
    if (int rc = mlstm_check(z, H, D, V, R)) return rc;
    ZLM_REQUIRE(max_new > 0 && scratch && (uintptr_t)scratch % 16 == 0, "mlstm: longest sequence %d", max_new);
    const MlstmGates gates{z, z_stride, i_off, f_off, VecW{bi, b_dtype}, VecW{bf, b_dtype}, cap};
    const int maxp = (max_new + ML_L - 1) / ML_L;
    const long long units = (long long)R * maxp * H, DV = (long long)D * V;
    ZLM_REQUIRE(units <= 2147483647LL && (D + 63) / 64 <= 65535 && (V + ML_COLS - 1) / ML_COLS <= 65535 && DV <= 65535LL * 128,
                "mlstm: %d sequences of up to %d tokens, heads of %d x %d", R, max_new, D, V);
    float2* part_m = (float2*)scratch;                        // [units] (b of the piece, the maximum it leaves by itself)
    float2* ahead = part_m + units;                           // [units] (maximum ahead, maximum after)
    float* part = (float*)(ahead + units);                    // [units][D][V], 16-byte aligned
    float* part_n = part + units * DV;                        // [units][D]
    const int esz = dtype == ZLM_DTYPE_BF16 ? 2 : 4;
    const int vec = (stride * esz) % 16 == 0 && (q_off * esz) % 16 == 0 && (k_off * esz) % 16 == 0 && (v_off * esz) % 16 == 0 &&
                    (D * esz) % 16 == 0 && (V * esz) % 16 == 0 && (uintptr_t)proj % 16 == 0;
    const size_t smem1 = (size_t)ML_L * (ML_LD + ML_COLS) * sizeof(float);
    const size_t smem3 = (size_t)(2 * ML_KC * ML_LD + ML_L * ML_LD + 2 * ML_KC * ML_COLS) * sizeof(float);
    const dim3 g1((unsigned)units, (D + 63) / 64, (V + ML_COLS - 1) / ML_COLS), g3((unsigned)units, (V + ML_COLS - 1) / ML_COLS);
#define ZLM_ML_RUN(TA)                                                                                                          \
    do {                                                                                                                        \
        static bool attr_set_dev[64] = {};                                                                                      \
        bool& attr_set = attr_set_dev[zlm_device_index()];                                                                      \
        if (!attr_set) {                                                                                                        \
            cudaError_t e1 = cudaFuncSetAttribute(mlstm_piece_kernel<TA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1); \
            cudaError_t e3 = cudaFuncSetAttribute(mlstm_out_kernel<TA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem3);   \
            if (e1 != cudaSuccess || e3 != cudaSuccess) {                                                                       \
                zlm_set_error("mlstm: cannot reserve shared memory");                                                           \
                return ZLM_ERR_CUDA;                                                                                            \
            }                                                                                                                   \
            attr_set = true;                                                                                                    \
        }                                                                                                                       \
        zlm_launch(mlstm_piece_kernel<TA>, g1, dim3(ML_THREADS), smem1, st, part, part_n, part_m, (const TA*)proj, stride, k_off, v_off, \
                   gates, seq_slot, cu_seqlens, H, D, V, maxp, vec);                                                            \
        if (DV % 4 == 0 && (uintptr_t)S % 16 == 0)                                                                              \
            zlm_launch(mlstm_chain_kernel<4>, dim3(R * H, (unsigned)((DV + 511) / 512)), dim3(128), 0, st, part, part_n,        \
                       (const float2*)part_m, ahead, S, n, (const float*)m, seq_slot, cu_seqlens, H, D, V, maxp);              \
        else                                                                                                                    \
            zlm_launch(mlstm_chain_kernel<1>, dim3(R * H, (unsigned)((DV + 127) / 128)), dim3(128), 0, st, part, part_n,        \
                       (const float2*)part_m, ahead, S, n, (const float*)m, seq_slot, cu_seqlens, H, D, V, maxp);              \
        zlm_launch(mlstm_out_kernel<TA>, g3, dim3(ML_THREADS), smem3, st, o, (const TA*)proj, stride, q_off, k_off, v_off, gates, \
                   (const float*)part, (const float*)part_n, (const float2*)ahead, m, seq_slot, cu_seqlens, H, D, V, maxp, q_scale, vec); \
    } while (0)
    if (dtype == ZLM_DTYPE_F32) {
        ZLM_ML_RUN(float);
    } else if (dtype == ZLM_DTYPE_BF16) {
        ZLM_ML_RUN(__nv_bfloat16);
    } else {
        ZLM_REQUIRE(false, "mlstm: unsupported dtype %d", dtype);
    }
#undef ZLM_ML_RUN
    return zlm_check_launch("mlstm");
}

ZLM_TRANSLATION_UNIT(mlstm)
