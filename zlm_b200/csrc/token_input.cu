// A layer's second look at its tokens: every token has, beside its row in the embedding, a row in a side table of which
// layer i owns `dim` columns.  The layer gates them by its stream and projects the result back:
//   g[t] = gelu_tanh(W_gate x[t]) * side[id_t, off : off + dim],   y = W_proj g   (y is normed and added to the stream)
// This file makes g, in two forms:
//   token_gate       elementwise, from W_gate x as a product of the library left it
//   token_gate_few   steps of up to 16 tokens, bf16 weights: the product (straight from the fp32 stream), the gelu and
//                    the row of the side table in one kernel
// Columns of g from dim up to g_cols become zeros.
#include "common.cuh"

__device__ __forceinline__ float ti_gelu_tanh(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <typename TA>
__global__ void __launch_bounds__(256)
token_gate_kernel(TA* __restrict__ g, int g_stride, int g_cols, const TA* __restrict__ z, int z_stride, const TA* __restrict__ side,
                  int side_stride, int off, const int* __restrict__ ids, int T, int dim, int V) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t n = (size_t)T * g_cols;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < n; e += (size_t)gridDim.x * blockDim.x) {
        const size_t t = e / g_cols;
        const int i = (int)(e - t * g_cols);
        TA* o = g + t * g_stride + i;
        if (!ZLM_CHK(o, sizeof(TA))) continue;
        float v = 0.f;
        if (i < dim && ZLM_CHK(ids + t, 4)) {
            const int id = min(max(ids[t], 0), V - 1);          // (validated on the host; a bad one never reads outside)
            const TA* zp = z + t * z_stride + i;
            const TA* sp = side + (size_t)id * side_stride + off + i;
            if (ZLM_CHK(zp, sizeof(TA)) && ZLM_CHK(sp, sizeof(TA))) v = ti_gelu_tanh(to_f32(*zp)) * to_f32(*sp);
        }
        *o = from_f32<TA>(v);
    }
}

extern "C" int zlm_token_gate(void* g, int g_stride, int g_cols, const void* z, int z_stride, const void* side, int side_stride,
                              int off, const int* ids, int dtype, int T, int dim, int V, cudaStream_t st) {
    if (T == 0) return ZLM_OK;
    ZLM_REQUIRE(T > 0 && dim > 0 && V > 0 && g_cols >= dim && g_stride >= g_cols && z_stride >= dim && off >= 0 && off + dim <= side_stride,
                "token_gate: %d columns from %d on of side rows of %d", dim, off, side_stride);
    const size_t n = (size_t)T * g_cols;
    const int blocks = (int)((n + 255) / 256 > 148 * 16 ? 148 * 16 : (n + 255) / 256);
    if (dtype == ZLM_DTYPE_F32)
        zlm_launch(token_gate_kernel<float>, blocks, 256, 0, st, (float*)g, g_stride, g_cols, (const float*)z, z_stride,
                   (const float*)side, side_stride, off, ids, T, dim, V);
    else if (dtype == ZLM_DTYPE_BF16)
        zlm_launch(token_gate_kernel<__nv_bfloat16>, blocks, 256, 0, st, (__nv_bfloat16*)g, g_stride, g_cols,
                   (const __nv_bfloat16*)z, z_stride, (const __nv_bfloat16*)side, side_stride, off, ids, T, dim, V);
    else
        ZLM_REQUIRE(false, "token_gate: unsupported dtype %d", dtype);
    return zlm_check_launch("token_gate");
}

// A block: TG_CH channels of the gate for all tokens; its warps share K (a lane eight neighbouring columns of every 2048),
// their sums meet in shared memory.  A sum's order depends on K alone.
#define TG_CH 4
#define TG_WARPS 8
#define TG_TOK 16
template <int TOK>
__global__ void __launch_bounds__(TG_WARPS * 32)
token_gate_few_kernel(__nv_bfloat16* __restrict__ g, int g_stride, int g_cols, const float* __restrict__ x,
                      const __nv_bfloat16* __restrict__ W, const __nv_bfloat16* __restrict__ side, int side_stride, int off,
                      const int* __restrict__ ids, int T, int K, int dim, int V) {
    __shared__ float part[TG_WARPS][TG_CH][TOK];
    pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c0 = blockIdx.x * TG_CH;
    float acc[TG_CH][TOK];
#pragma unroll
    for (int c = 0; c < TG_CH; ++c)
#pragma unroll
        for (int t = 0; t < TOK; ++t) acc[c][t] = 0.f;
    bool waited = false;
    for (int k = (warp * 32 + lane) * 8; k < K; k += TG_WARPS * 256) {
        uint4 w[TG_CH];
#pragma unroll
        for (int c = 0; c < TG_CH; ++c) {
            const __nv_bfloat16* wp = W + (size_t)(c0 + c) * K + k;
            w[c] = (c0 + c < dim && ZLM_CHK(wp, 16)) ? *(const uint4*)wp : make_uint4(0u, 0u, 0u, 0u);
        }
        if (!waited) {              // the weights do not change during a step: only the stream has to be waited for
            pdl_wait();
            waited = true;
        }
#pragma unroll
        for (int t = 0; t < TOK; ++t) {
            if (t >= T) break;
            const float* xp = x + (size_t)t * K + k;
            if (!ZLM_CHK(xp, 32)) continue;
            const float4 a = *(const float4*)xp, b = *(const float4*)(xp + 4);
#pragma unroll
            for (int c = 0; c < TG_CH; ++c) {
                float s = acc[c][t];
                s = fmaf(__uint_as_float(w[c].x << 16), a.x, s); s = fmaf(__uint_as_float(w[c].x & 0xffff0000u), a.y, s);
                s = fmaf(__uint_as_float(w[c].y << 16), a.z, s); s = fmaf(__uint_as_float(w[c].y & 0xffff0000u), a.w, s);
                s = fmaf(__uint_as_float(w[c].z << 16), b.x, s); s = fmaf(__uint_as_float(w[c].z & 0xffff0000u), b.y, s);
                s = fmaf(__uint_as_float(w[c].w << 16), b.z, s); s = fmaf(__uint_as_float(w[c].w & 0xffff0000u), b.w, s);
                acc[c][t] = s;
            }
        }
    }
    if (!waited) pdl_wait();
#pragma unroll
    for (int c = 0; c < TG_CH; ++c)
#pragma unroll
        for (int t = 0; t < TOK; ++t) {
            const float s = warp_sum(acc[c][t]);
            if (lane == 0) part[warp][c][t] = s;
        }
    __syncthreads();
    const int c = threadIdx.x % TG_CH, t = threadIdx.x / TG_CH;
    if (t >= T || t >= TOK || c0 + c >= g_cols) return;
    float v = 0.f;
    if (c0 + c < dim && ZLM_CHK(ids + t, 4)) {
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < TG_WARPS; ++w) s += part[w][c][t];
        const int id = min(max(ids[t], 0), V - 1);
        const __nv_bfloat16* sp = side + (size_t)id * side_stride + off + c0 + c;
        if (ZLM_CHK(sp, 2)) v = ti_gelu_tanh(s) * to_f32(*sp);
    }
    __nv_bfloat16* o = g + (size_t)t * g_stride + c0 + c;
    if (ZLM_CHK(o, 2)) *o = __float2bfloat16_rn(v);
}

// 1 if the fused form takes the step
extern "C" int zlm_token_gate_few_supported(int T, int K) { return (T >= 1 && T <= TG_TOK && K % 8 == 0) ? 1 : 0; }

extern "C" int zlm_token_gate_few(void* g, int g_stride, int g_cols, const float* x, const void* W, const void* side, int side_stride,
                                  int off, const int* ids, int T, int K, int dim, int V, cudaStream_t st) {
    if (T == 0) return ZLM_OK;
    ZLM_REQUIRE(zlm_token_gate_few_supported(T, K), "token_gate_few: T=%d K=%d", T, K);
    ZLM_REQUIRE(dim > 0 && V > 0 && g_cols >= dim && g_stride >= g_cols && off >= 0 && off + dim <= side_stride,
                "token_gate_few: %d columns from %d on of side rows of %d", dim, off, side_stride);
    ZLM_REQUIRE((uintptr_t)x % 16 == 0 && (uintptr_t)W % 16 == 0, "token_gate_few: stream and weights must be 16-byte aligned");
    const int blocks = (g_cols + TG_CH - 1) / TG_CH;
#define ZLM_TG(TOK)                                                                                                         \
    zlm_launch(token_gate_few_kernel<TOK>, blocks, TG_WARPS * 32, 0, st, (__nv_bfloat16*)g, g_stride, g_cols, x,                \
               (const __nv_bfloat16*)W, (const __nv_bfloat16*)side, side_stride, off, ids, T, K, dim, V)
    if (T <= 1) ZLM_TG(1);
    else if (T <= 4) ZLM_TG(4);
    else if (T <= 8) ZLM_TG(8);
    else ZLM_TG(16);
#undef ZLM_TG
    return zlm_check_launch("token_gate_few");
}

ZLM_TRANSLATION_UNIT(token_input)
