// A gated recurrence whose gates read the current token alone (minGRU), one number of state per channel:
//   z = sigmoid(zp + bz),  u = xp + bx,  cand = u + 1/2 where u >= 0, sigmoid(u) where u < 0
//   S_t = (1 - z) S_(t-1) + z cand,  out = S_t silu(gp)
// zp, xp, gp are W columns each of one projection.  Gates, candidate, state and read-out are fp32 in both element types.
// A sequence's state is a row of [slots][W] fp32, read at a step's start and written at its end (zeros in a new slot).
//
// Short steps: a thread walks the step's tokens of its channels.  Long ones run in pieces of GRU_PIECE tokens side by
// side: what a piece does to a state, S_out = A S_in + B, is gathered piece by piece, the pieces are chained, and every
// piece walks its tokens again from the state it really starts from.  1 - z is formed as sigmoid(-(zp + bz)).
#include "common.cuh"

#define GRU_PIECE 32
#define GRU_AHEAD 16            // tokens whose loads are in flight in the pieces' walks
#define GRU_SHORT_AHEAD 8

// VEC neighbouring elements of a row as floats, and back
template <typename TA, int VEC> __device__ __forceinline__ void gru_load(const TA* p, float* f) {
    if (VEC == 1) {
        f[0] = to_f32(p[0]);
    } else if (sizeof(TA) == 2) {
        const unsigned u = *(const unsigned*)p;
        f[0] = __uint_as_float(u << 16);
        f[1] = __uint_as_float(u & 0xffff0000u);
    } else {
        const float2 v = *(const float2*)p;
        f[0] = v.x;
        f[1] = v.y;
    }
}
template <typename TA, int VEC> __device__ __forceinline__ void gru_store(TA* p, const float* f) {
    if (VEC == 1) {
        p[0] = from_f32<TA>(f[0]);
    } else if (sizeof(TA) == 2) {
        *(__nv_bfloat162*)p = __floats2bfloat162_rn(f[0], f[1]);
    } else {
        *(float2*)p = make_float2(f[0], f[1]);
    }
}

// a token's decay a = 1 - z and input b = z * cand
__device__ __forceinline__ void gru_ab(float z, float u, float& a, float& b) {
    const float e = expf(-fabsf(z)), lo = e / (1.0f + e), hi = 1.0f / (1.0f + e);      // sigmoid(-|z|), sigmoid(|z|)
    a = z >= 0.f ? lo : hi;
    const float cand = u >= 0.f ? u + 0.5f : 1.0f / (1.0f + expf(-u));
    b = (z >= 0.f ? hi : lo) * cand;
}
__device__ __forceinline__ float gru_silu(float g) { return g / (1.0f + expf(-g)); }

// One walk over tokens [lo, hi) of the sequence whose rows start at row0, from state S: with OUT the outputs are
// written; without, A and B gather what the walk does to a state.
template <typename TA, int VEC, int AHEAD, bool OUT>
__device__ __forceinline__ void gru_walk(float* S, float* A, const TA* __restrict__ proj, int stride, int z_off, int x_off,
                                         int g_off, const float* zb, const float* xb, TA* __restrict__ out, int out_stride, int c,
                                         int row0, int lo, int hi) {
    for (int s0 = lo; s0 < hi; s0 += AHEAD) {
        float z[AHEAD][VEC], u[AHEAD][VEC], g[OUT ? AHEAD : 1][VEC];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const TA* p = proj + (size_t)(row0 + s0 + j) * stride + c;
            const bool ok = s0 + j < hi && ZLM_CHK(p + z_off, VEC * sizeof(TA)) && ZLM_CHK(p + x_off, VEC * sizeof(TA)) &&
                            (!OUT || ZLM_CHK(p + g_off, VEC * sizeof(TA)));
            if (ok) {
                gru_load<TA, VEC>(p + z_off, z[j]);
                gru_load<TA, VEC>(p + x_off, u[j]);
                if (OUT) gru_load<TA, VEC>(p + g_off, g[j]);
            } else {
#pragma unroll
                for (int v = 0; v < VEC; ++v) {
                    z[j][v] = u[j][v] = 0.f;
                    if (OUT) g[j][v] = 0.f;
                }
            }
        }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (s0 + j >= hi) break;
            float y[VEC];
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                float a, b;
                gru_ab(z[j][v] + zb[v], u[j][v] + xb[v], a, b);
                S[v] = fmaf(a, S[v], b);
                if (OUT) y[v] = S[v] * gru_silu(g[j][v]);
                else A[v] *= a;
            }
            if (OUT) {
                TA* o = out + (size_t)(row0 + s0 + j) * out_stride + c;
                if (ZLM_CHK(o, VEC * sizeof(TA))) gru_store<TA, VEC>(o, y);
            }
        }
    }
}

template <int VEC> __device__ __forceinline__ void gru_biases(const VecW& bz, const VecW& bx, int c, float* zb, float* xb) {
#pragma unroll
    for (int v = 0; v < VEC; ++v) {
        zb[v] = bz.p ? bz[c + v] : 0.f;
        xb[v] = bx.p ? bx[c + v] : 0.f;
    }
}

template <typename TA, int VEC>
__global__ void __launch_bounds__(128)
mingru_scan_kernel(TA* __restrict__ out, int out_stride, const TA* __restrict__ proj, int stride, int z_off, int x_off, int g_off,
                   VecW bz, VecW bx, float* __restrict__ state, const int* __restrict__ seq_slot,
                   const int* __restrict__ cu_seqlens, int W) {
    pdl_trigger();
    const int r = blockIdx.x, c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    if (c >= W) return;
    float zb[VEC], xb[VEC], S[VEC];
    gru_biases<VEC>(bz, bx, c, zb, xb);
    pdl_wait();
    if (!ZLM_CHK(seq_slot + r, 4) || !ZLM_CHK(cu_seqlens + r, 8)) return;
    const int row0 = cu_seqlens[r], n = cu_seqlens[r + 1] - row0;
    float* sp = state + (size_t)seq_slot[r] * W + c;
    if (!ZLM_CHK(sp, VEC * 4)) return;
#pragma unroll
    for (int v = 0; v < VEC; ++v) S[v] = sp[v];
    gru_walk<TA, VEC, GRU_SHORT_AHEAD, true>(S, nullptr, proj, stride, z_off, x_off, g_off, zb, xb, out, out_stride, c, row0, 0, n);
#pragma unroll
    for (int v = 0; v < VEC; ++v) sp[v] = S[v];
}

// what every piece does to a state: PA [R][maxp][W] the product of its decays, PB its state from zero
template <typename TA, int VEC>
__global__ void __launch_bounds__(128)
mingru_piece_kernel(float* __restrict__ PA, float* __restrict__ PB, const TA* __restrict__ proj, int stride, int z_off, int x_off,
                    VecW bz, VecW bx, const int* __restrict__ cu_seqlens, int W, int maxp) {
    pdl_trigger();
    const int r = blockIdx.x / maxp, p = blockIdx.x % maxp, c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    pdl_wait();
    if (c >= W || !ZLM_CHK(cu_seqlens + r, 8)) return;
    const int row0 = cu_seqlens[r], n = cu_seqlens[r + 1] - row0;
    const int lo = p * GRU_PIECE, hi = min(n, lo + GRU_PIECE);
    if (lo >= hi) return;
    float zb[VEC], xb[VEC], S[VEC], A[VEC];
    gru_biases<VEC>(bz, bx, c, zb, xb);
#pragma unroll
    for (int v = 0; v < VEC; ++v) { S[v] = 0.f; A[v] = 1.f; }
    gru_walk<TA, VEC, GRU_AHEAD, false>(S, A, proj, stride, z_off, x_off, 0, zb, xb, nullptr, 0, c, row0, lo, hi);
    const size_t at = ((size_t)r * maxp + p) * W + c;
    if (!ZLM_CHK(PA + at, VEC * 4) || !ZLM_CHK(PB + at, VEC * 4)) return;
#pragma unroll
    for (int v = 0; v < VEC; ++v) { PA[at + v] = A[v]; PB[at + v] = S[v]; }
}

// the pieces in order: PA[piece] becomes the state the piece starts from; the sequence's state is left
__global__ void __launch_bounds__(128)
mingru_chain_kernel(float* __restrict__ PA, const float* __restrict__ PB, float* __restrict__ state,
                    const int* __restrict__ seq_slot, const int* __restrict__ cu_seqlens, int W, int maxp) {
    pdl_trigger();
    const int r = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    pdl_wait();
    if (c >= W || !ZLM_CHK(seq_slot + r, 4) || !ZLM_CHK(cu_seqlens + r, 8)) return;
    const int n = cu_seqlens[r + 1] - cu_seqlens[r], np = (n + GRU_PIECE - 1) / GRU_PIECE;
    float* sp = state + (size_t)seq_slot[r] * W + c;
    if (!ZLM_CHK(sp, 4)) return;
    float S = *sp;
    for (int p0 = 0; p0 < np; p0 += GRU_AHEAD) {
        float A[GRU_AHEAD], B[GRU_AHEAD];
#pragma unroll
        for (int j = 0; j < GRU_AHEAD; ++j) {
            const size_t at = ((size_t)r * maxp + p0 + j) * W + c;
            const bool ok = p0 + j < np && ZLM_CHK(PA + at, 4) && ZLM_CHK(PB + at, 4);
            A[j] = ok ? PA[at] : 1.f;
            B[j] = ok ? PB[at] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < GRU_AHEAD; ++j) {
            if (p0 + j >= np) break;
            const size_t at = ((size_t)r * maxp + p0 + j) * W + c;
            if (ZLM_CHK(PA + at, 4)) PA[at] = S;
            S = fmaf(A[j], S, B[j]);
        }
    }
    *sp = S;
}

template <typename TA, int VEC>
__global__ void __launch_bounds__(128)
mingru_piece_out_kernel(TA* __restrict__ out, int out_stride, const TA* __restrict__ proj, int stride, int z_off, int x_off,
                        int g_off, VecW bz, VecW bx, const float* __restrict__ S0, const int* __restrict__ cu_seqlens, int W,
                        int maxp) {
    pdl_trigger();
    const int r = blockIdx.x / maxp, p = blockIdx.x % maxp, c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    pdl_wait();
    if (c >= W || !ZLM_CHK(cu_seqlens + r, 8)) return;
    const int row0 = cu_seqlens[r], n = cu_seqlens[r + 1] - row0;
    const int lo = p * GRU_PIECE, hi = min(n, lo + GRU_PIECE);
    if (lo >= hi) return;
    const size_t at = ((size_t)r * maxp + p) * W + c;
    if (!ZLM_CHK(S0 + at, VEC * 4)) return;
    float zb[VEC], xb[VEC], S[VEC];
    gru_biases<VEC>(bz, bx, c, zb, xb);
#pragma unroll
    for (int v = 0; v < VEC; ++v) S[v] = S0[at + v];
    gru_walk<TA, VEC, GRU_SHORT_AHEAD, true>(S, nullptr, proj, stride, z_off, x_off, g_off, zb, xb, out, out_stride, c, row0, lo, hi);
}

template <typename TA, int VEC>
static void launch_mingru(void* out, int out_stride, const void* proj, int stride, int z_off, int x_off, int g_off, VecW bz, VecW bx,
                          float* state, const int* seq_slot, const int* cu_seqlens, int R, int W, int max_new, float* pieces,
                          cudaStream_t st) {
    const int per = 128 * VEC, cols = (W + per - 1) / per;
    if (!pieces) {
        zlm_launch(mingru_scan_kernel<TA, VEC>, dim3(R, cols), dim3(128), 0, st, (TA*)out, out_stride, (const TA*)proj, stride, z_off,
                   x_off, g_off, bz, bx, state, seq_slot, cu_seqlens, W);
        return;
    }
    const int maxp = (max_new + GRU_PIECE - 1) / GRU_PIECE;
    float* PA = pieces;
    float* PB = pieces + (size_t)R * maxp * W;
    zlm_launch(mingru_piece_kernel<TA, VEC>, dim3(R * maxp, cols), dim3(128), 0, st, PA, PB, (const TA*)proj, stride, z_off, x_off, bz,
               bx, cu_seqlens, W, maxp);
    zlm_launch(mingru_chain_kernel, dim3(R, (W + 127) / 128), dim3(128), 0, st, PA, (const float*)PB, state, seq_slot, cu_seqlens, W,
               maxp);
    zlm_launch(mingru_piece_out_kernel<TA, VEC>, dim3(R * maxp, cols), dim3(128), 0, st, (TA*)out, out_stride, (const TA*)proj, stride,
               z_off, x_off, g_off, bz, bx, (const float*)PA, cu_seqlens, W, maxp);
}

// proj [T][stride] holds zp, xp and gp from columns z_off, x_off, g_off on (W columns each, without the biases bz, bx [W],
// which may be null); state [slots][W] fp32; out [T][out_stride].  pieces: null (a thread walks a sequence's tokens), or
// 2 * R * ceil(max_new / 32) * W floats: sequences run in pieces of 32 tokens side by side.
extern "C" int zlm_mingru(void* out, int out_stride, const void* proj, int stride, int z_off, int x_off, int g_off, const void* bz,
                          const void* bx, int bias_dtype, float* state, int dtype, const int* seq_slot, const int* cu_seqlens, int T,
                          int R, int W, int max_new, float* pieces, cudaStream_t st) {
    if (T == 0) return ZLM_OK;
    ZLM_REQUIRE(T > 0 && R > 0 && W > 0 && out_stride >= W && (W + 127) / 128 <= 65535, "mingru: bad sizes T=%d sequences=%d channels=%d",
                T, R, W);
    ZLM_REQUIRE(z_off >= 0 && x_off >= 0 && g_off >= 0 && z_off + W <= stride && x_off + W <= stride && g_off + W <= stride,
                "mingru: columns %d, %d, %d of %d channels in rows of %d", z_off, x_off, g_off, W, stride);
    ZLM_REQUIRE(!pieces || max_new > 0, "mingru: pieces of a longest sequence of %d", max_new);
    const VecW vz{bz, bias_dtype}, vx{bx, bias_dtype};
    const size_t pair = dtype == ZLM_DTYPE_F32 ? 8 : 4;
    const bool vec = W % 2 == 0 && stride % 2 == 0 && out_stride % 2 == 0 && z_off % 2 == 0 && x_off % 2 == 0 && g_off % 2 == 0 &&
                     (uintptr_t)proj % pair == 0 && (uintptr_t)out % pair == 0;
#define ZLM_GRU(TA, VEC)                                                                                                        \
    launch_mingru<TA, VEC>(out, out_stride, proj, stride, z_off, x_off, g_off, vz, vx, state, seq_slot, cu_seqlens, R, W, max_new, \
                           pieces, st)
    if (dtype == ZLM_DTYPE_F32) {
        if (vec) ZLM_GRU(float, 2); else ZLM_GRU(float, 1);
    } else if (dtype == ZLM_DTYPE_BF16) {
        if (vec) ZLM_GRU(__nv_bfloat16, 2); else ZLM_GRU(__nv_bfloat16, 1);
    } else {
        ZLM_REQUIRE(false, "mingru: unsupported dtype %d", dtype);
    }
#undef ZLM_GRU
    return zlm_check_launch("mingru");
}

ZLM_TRANSLATION_UNIT(mingru)
