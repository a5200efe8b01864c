// A gated recurrence whose gates read the current token alone (minGRU), one number of state per channel:
//   z = sigmoid(zp + bz),  u = xp + bx,  cand = u + 1/2 where u >= 0, sigmoid(u) where u < 0
//   S_t = (1 - z) S_(t-1) + z cand,  out = S_t silu(gp)
// zp, xp, gp are W columns each of one projection.  Gates, candidate, state and read-out are fp32 in both element types.
// A sequence's state is a row of [slots][W] fp32, read at a step's start and written at its end (zeros in a new slot).
//
// Short steps: a thread walks the step's tokens of its channels.  Long ones run on thread-block clusters: a cluster of
// GRU_CLUSTER blocks owns a strip of channels of one sequence, every warp a piece of P neighbouring tokens, whose gates and
// candidates it keeps in registers.  What a piece does to a state, S_out = A S_in + B, is folded over the block's warps in
// shared memory and over the cluster's blocks through distributed shared memory; then every warp knows the state its piece
// starts from and walks it, so the projection is read once.  A sequence of more than GRU_CLUSTER x GRU_WARPS x P tokens goes
// round again from the state the cluster ends with.  1 - z is formed as sigmoid(-(zp + bz)).
#include "common.cuh"
#include <cooperative_groups.h>
namespace cg = cooperative_groups;

#define GRU_SHORT_AHEAD 8
#define GRU_CLUSTER 8
#define GRU_WARPS 8

// VEC neighbouring elements of a row, as they are stored
template <typename TA, int VEC> struct GruRaw { TA v[VEC]; };
template <> struct GruRaw<__nv_bfloat16, 2> { unsigned v; };
template <> struct GruRaw<float, 2> { float2 v; };
template <typename TA, int VEC> __device__ __forceinline__ GruRaw<TA, VEC> gru_load(const TA* p) {
    return *reinterpret_cast<const GruRaw<TA, VEC>*>(p);
}
__device__ __forceinline__ float gru_get(const GruRaw<__nv_bfloat16, 2>& r, int i) {
    return __uint_as_float(i ? (r.v & 0xffff0000u) : (r.v << 16));
}
__device__ __forceinline__ float gru_get(const GruRaw<float, 2>& r, int i) { return i ? r.v.y : r.v.x; }
template <typename TA> __device__ __forceinline__ float gru_get(const GruRaw<TA, 1>& r, int) { return to_f32(r.v[0]); }
template <typename TA, int VEC> __device__ __forceinline__ GruRaw<TA, VEC> gru_zero() {
    GruRaw<TA, VEC> r;
    memset(&r, 0, sizeof(r));
    return r;
}
template <typename TA, int VEC> __device__ __forceinline__ void gru_store(TA* p, const float* f) {
    if (VEC == 1) {
        p[0] = from_f32<TA>(f[0]);
    } else if (sizeof(TA) == 2) {
        *(__nv_bfloat162*)p = __floats2bfloat162_rn(f[0], f[VEC - 1]);
    } else {
        *(float2*)p = make_float2(f[0], f[VEC - 1]);
    }
}

// e^x and 1 / x: the 32-bit path takes the library's, the bfloat16 path the fast forms (a few units of the last place of
// fp32, far below the rounding of what goes in and comes out)
template <bool FAST> __device__ __forceinline__ float gru_exp(float x) { return FAST ? __expf(x) : expf(x); }
template <bool FAST> __device__ __forceinline__ float gru_inv(float x) { return FAST ? __fdividef(1.0f, x) : 1.0f / x; }

// a token's decay a = 1 - z and input b = z * cand
template <bool FAST> __device__ __forceinline__ void gru_ab(float z, float u, float& a, float& b) {
    const float e = gru_exp<FAST>(-fabsf(z)), hi = gru_inv<FAST>(1.0f + e), lo = e * hi;      // sigmoid(|z|), sigmoid(-|z|)
    a = z >= 0.f ? lo : hi;
    const float cand = u >= 0.f ? u + 0.5f : gru_inv<FAST>(1.0f + gru_exp<FAST>(-u));
    b = (z >= 0.f ? hi : lo) * cand;
}
template <bool FAST> __device__ __forceinline__ float gru_silu(float g) { return g * gru_inv<FAST>(1.0f + gru_exp<FAST>(-g)); }

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
    constexpr bool FAST = sizeof(TA) == 2;
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
    for (int s0 = 0; s0 < n; s0 += GRU_SHORT_AHEAD) {
        GruRaw<TA, VEC> z[GRU_SHORT_AHEAD], u[GRU_SHORT_AHEAD], g[GRU_SHORT_AHEAD];
#pragma unroll
        for (int j = 0; j < GRU_SHORT_AHEAD; ++j) {
            const TA* p = proj + (size_t)(row0 + s0 + j) * stride + c;
            const bool ok = s0 + j < n && ZLM_CHK(p + z_off, VEC * sizeof(TA)) && ZLM_CHK(p + x_off, VEC * sizeof(TA)) &&
                            ZLM_CHK(p + g_off, VEC * sizeof(TA));
            z[j] = ok ? gru_load<TA, VEC>(p + z_off) : gru_zero<TA, VEC>();
            u[j] = ok ? gru_load<TA, VEC>(p + x_off) : gru_zero<TA, VEC>();
            g[j] = ok ? gru_load<TA, VEC>(p + g_off) : gru_zero<TA, VEC>();
        }
#pragma unroll
        for (int j = 0; j < GRU_SHORT_AHEAD; ++j) {
            if (s0 + j >= n) break;
            float y[VEC];
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                float a, b;
                gru_ab<FAST>(gru_get(z[j], v) + zb[v], gru_get(u[j], v) + xb[v], a, b);
                S[v] = fmaf(a, S[v], b);
                y[v] = S[v] * gru_silu<FAST>(gru_get(g[j], v));
            }
            TA* o = out + (size_t)(row0 + s0 + j) * out_stride + c;
            if (ZLM_CHK(o, VEC * sizeof(TA))) gru_store<TA, VEC>(o, y);
        }
    }
#pragma unroll
    for (int v = 0; v < VEC; ++v) sp[v] = S[v];
}

template <typename TA, int VEC, int P>
__global__ void __cluster_dims__(GRU_CLUSTER, 1, 1) __launch_bounds__(GRU_WARPS * 32, 2)
mingru_cluster_kernel(TA* __restrict__ out, int out_stride, const TA* __restrict__ proj, int stride, int z_off, int x_off,
                      int g_off, VecW bz, VecW bx, float* __restrict__ state, const int* __restrict__ seq_slot,
                      const int* __restrict__ cu_seqlens, int W) {
    constexpr bool FAST = sizeof(TA) == 2;
    constexpr int CH = 32 * VEC;
    // two sets, for rounds in turn: a block that is a round ahead does not overwrite what another still reads
    __shared__ float2 piece[2][GRU_WARPS][CH];
    __shared__ float2 total[2][CH];
    cg::cluster_group cluster = cg::this_cluster();
    const int rank = (int)cluster.block_rank(), r = blockIdx.x / GRU_CLUSTER;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int c = blockIdx.y * CH + lane * VEC;
    pdl_trigger();
    bool live = c < W;                               // (no thread leaves early: the cluster meets at barriers)
    float zb[VEC], xb[VEC], S0[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) zb[v] = xb[v] = S0[v] = 0.f;
    if (live) gru_biases<VEC>(bz, bx, c, zb, xb);
    pdl_wait();
    int row0 = 0, n = 0, slot = 0;
    if (ZLM_CHK(seq_slot + r, 4) && ZLM_CHK(cu_seqlens + r, 8)) {
        row0 = cu_seqlens[r];
        n = cu_seqlens[r + 1] - row0;
        slot = seq_slot[r];
    }
    float* sp = state + (size_t)slot * W + c;
    live = live && ZLM_CHK(sp, VEC * 4);
    if (live)
#pragma unroll
        for (int v = 0; v < VEC; ++v) S0[v] = sp[v];
    int par = 0;
    for (int base = 0; base < n; base += GRU_CLUSTER * GRU_WARPS * P, par ^= 1) {
        const int lo = base + (rank * GRU_WARPS + warp) * P, cnt = live ? min(n - lo, P) : 0;
        GruRaw<TA, VEC> z[P], u[P], g[P];
#pragma unroll
        for (int j = 0; j < P; ++j) {
            const TA* p = proj + (size_t)(row0 + lo + j) * stride + c;
            const bool ok = j < cnt && ZLM_CHK(p + z_off, VEC * sizeof(TA)) && ZLM_CHK(p + x_off, VEC * sizeof(TA)) &&
                            ZLM_CHK(p + g_off, VEC * sizeof(TA));
            z[j] = ok ? gru_load<TA, VEC>(p + z_off) : gru_zero<TA, VEC>();
            u[j] = ok ? gru_load<TA, VEC>(p + x_off) : gru_zero<TA, VEC>();
            g[j] = ok ? gru_load<TA, VEC>(p + g_off) : gru_zero<TA, VEC>();
        }
        float a[P][VEC], b[P][VEC], A[VEC], B[VEC];
#pragma unroll
        for (int v = 0; v < VEC; ++v) { A[v] = 1.f; B[v] = 0.f; }
#pragma unroll
        for (int j = 0; j < P; ++j)
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                gru_ab<FAST>(gru_get(z[j], v) + zb[v], gru_get(u[j], v) + xb[v], a[j][v], b[j][v]);
                if (j < cnt) {
                    A[v] *= a[j][v];
                    B[v] = fmaf(a[j][v], B[v], b[j][v]);
                }
            }
#pragma unroll
        for (int v = 0; v < VEC; ++v) piece[par][warp][lane * VEC + v] = make_float2(A[v], B[v]);
        __syncthreads();
        if (warp == 0)
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                float2 t = piece[par][0][lane * VEC + v];
                for (int w = 1; w < GRU_WARPS; ++w) {
                    const float2 q = piece[par][w][lane * VEC + v];
                    t = make_float2(q.x * t.x, fmaf(q.x, t.y, q.y));
                }
                total[par][lane * VEC + v] = t;
            }
        cluster.sync();
        // the state this warp's piece starts from, and the one the whole round ends with
        float S[VEC];
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
            float2 t[GRU_CLUSTER];
#pragma unroll
            for (int k = 0; k < GRU_CLUSTER; ++k) t[k] = cluster.map_shared_rank(&total[par][0], k)[lane * VEC + v];
            float s = S0[v];
            S[v] = s;
#pragma unroll
            for (int k = 0; k < GRU_CLUSTER; ++k) {
                s = fmaf(t[k].x, s, t[k].y);
                if (k + 1 == rank) S[v] = s;
            }
            S0[v] = s;
            for (int w = 0; w < warp; ++w) {
                const float2 q = piece[par][w][lane * VEC + v];
                S[v] = fmaf(q.x, S[v], q.y);
            }
        }
#pragma unroll
        for (int j = 0; j < P; ++j) {
            if (j >= cnt) break;
            float y[VEC];
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                S[v] = fmaf(a[j][v], S[v], b[j][v]);
                y[v] = S[v] * gru_silu<FAST>(gru_get(g[j], v));
            }
            TA* o = out + (size_t)(row0 + lo + j) * out_stride + c;
            if (ZLM_CHK(o, VEC * sizeof(TA))) gru_store<TA, VEC>(o, y);
        }
    }
    if (live && rank == 0 && warp == 0)              // (every block has read the old state ahead of the first barrier)
#pragma unroll
        for (int v = 0; v < VEC; ++v) sp[v] = S0[v];
    cluster.sync();                                  // no block leaves while another may still read its shared memory
}

template <typename TA, int VEC>
static void launch_mingru(void* out, int out_stride, const void* proj, int stride, int z_off, int x_off, int g_off, VecW bz, VecW bx,
                          float* state, const int* seq_slot, const int* cu_seqlens, int R, int W, int cluster, cudaStream_t st) {
    if (!cluster) {
        zlm_launch(mingru_scan_kernel<TA, VEC>, dim3(R, (W + 128 * VEC - 1) / (128 * VEC)), dim3(128), 0, st, (TA*)out, out_stride,
                   (const TA*)proj, stride, z_off, x_off, g_off, bz, bx, state, seq_slot, cu_seqlens, W);
        return;
    }
    constexpr int P = sizeof(TA) == 4 && VEC == 2 ? 8 : 16;
    zlm_launch(mingru_cluster_kernel<TA, VEC, P>, dim3(R * GRU_CLUSTER, (W + 32 * VEC - 1) / (32 * VEC)), dim3(GRU_WARPS * 32), 0, st,
               (TA*)out, out_stride, (const TA*)proj, stride, z_off, x_off, g_off, bz, bx, state, seq_slot, cu_seqlens, W);
}

// proj [T][stride] holds zp, xp and gp from columns z_off, x_off, g_off on (W columns each, without the biases bz, bx [W],
// which may be null); state [slots][W] fp32; out [T][out_stride].  cluster 0: a thread walks a sequence's tokens; 1: a
// cluster of blocks shares them.
extern "C" int zlm_mingru(void* out, int out_stride, const void* proj, int stride, int z_off, int x_off, int g_off, const void* bz,
                          const void* bx, int bias_dtype, float* state, int dtype, const int* seq_slot, const int* cu_seqlens, int T,
                          int R, int W, int cluster, cudaStream_t st) {
    if (T == 0) return ZLM_OK;
    ZLM_REQUIRE(T > 0 && R > 0 && W > 0 && out_stride >= W && (W + 31) / 32 <= 65535, "mingru: bad sizes T=%d sequences=%d channels=%d",
                T, R, W);
    ZLM_REQUIRE(z_off >= 0 && x_off >= 0 && g_off >= 0 && z_off + W <= stride && x_off + W <= stride && g_off + W <= stride,
                "mingru: columns %d, %d, %d of %d channels in rows of %d", z_off, x_off, g_off, W, stride);
    const VecW vz{bz, bias_dtype}, vx{bx, bias_dtype};
    const size_t pair = dtype == ZLM_DTYPE_F32 ? 8 : 4;
    const bool vec = W % 2 == 0 && stride % 2 == 0 && out_stride % 2 == 0 && z_off % 2 == 0 && x_off % 2 == 0 && g_off % 2 == 0 &&
                     (uintptr_t)proj % pair == 0 && (uintptr_t)out % pair == 0;
#define ZLM_GRU(TA, VEC)                                                                                                        \
    launch_mingru<TA, VEC>(out, out_stride, proj, stride, z_off, x_off, g_off, vz, vx, state, seq_slot, cu_seqlens, R, W, cluster, st)
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
