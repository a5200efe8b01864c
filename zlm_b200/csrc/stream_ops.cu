// Operations on the fp32 residual stream and around it that designs with a norm on the sublayer's *output* need:
//   embed_scaled     out[t] = table[id_t] * scale (+ pair[(id_(t-1) * mul_prev + id_t * mul_cur) mod buckets], a second
//                    table looked up by the token and the token before it; the row `buckets` for a sequence's first
//                    token).  The token before a step's first one is per-slot state.
//   norm_scale_add   stream[t] += y[t] / sqrt(mean(y[t]^2) + eps) * w (* ls): RMS norm of a sublayer's output, an
//                    optional second vector (a scale per coordinate of the layer), and the residual add, all in fp32
//   norm_add_norm    the same (without ls) and the norm, RMS or layer norm, that reads the stream next; in a step of one
//                    token a sequence also that layer's convolution over time of the normed rows
//   poly_norm        a polynomial of normed powers as a feed-forward's activation
//   cast_rows        the stream's rows rounded to the compute dtype (the input of a sublayer that reads the stream
//                    itself, without a norm before it)
//   gated_act        out[t, i] = act(gu[t, i]) * gu[t, I + i], act = silu or the tanh form of gelu
//   scale_f32        x *= s (logits times a constant)
//   head_scalar_gate x[t, h, :] *= sigmoid(g[t, h]): one gate number per head
#include "common.cuh"
#include "elementwise.cuh"

// ---------------------------------------------------------------- embedding with a scale and a pair table
template <typename TW>
__global__ void embed_scaled_kernel(float* __restrict__ out, const TW* __restrict__ table, float scale,
                                    const TW* __restrict__ pair, int buckets, long long mul_prev, long long mul_cur,
                                    const int* __restrict__ ids, const int* __restrict__ token_pos,
                                    const int* __restrict__ token_seq, const int* __restrict__ cu_seqlens,
                                    const int* __restrict__ seq_slot, int* __restrict__ prev_state, int H, int V) {
    __shared__ int s_row;
    pdl_trigger();
    const int t = blockIdx.x;
    pdl_wait();                 // the ids may be what the previous step's sampler wrote
    if (!ZLM_CHK(ids + t, 4) || !ZLM_CHK(out + (size_t)t * H, (size_t)H * 4)) return;
    int id = ids[t];
    id = id < 0 ? 0 : (id >= V ? V - 1 : id);       // ids are validated on the host; a bad one never reads outside
    if (pair != nullptr && threadIdx.x == 0) {
        int row = buckets;
        if (ZLM_CHK(token_pos + t, 4) && ZLM_CHK(token_seq + t, 4)) {
            const int seq = token_seq[t];
            if (ZLM_CHK(cu_seqlens + seq, 8) && ZLM_CHK(seq_slot + seq, 4)) {
                const int first = cu_seqlens[seq], last = cu_seqlens[seq + 1] - 1;
                const int slot = seq_slot[seq];
                int prev = -1;
                if (t > first) {
                    prev = ZLM_CHK(ids + t - 1, 4) ? ids[t - 1] : -1;
                } else {
                    // the step's first token of this sequence: the token before it is the slot's state, which this
                    // same thread then replaces by the step's last token (nobody else reads or writes it)
                    if (token_pos[t] > 0 && ZLM_CHK(prev_state + slot, 4)) prev = prev_state[slot];
                    if (ZLM_CHK(prev_state + slot, 4) && ZLM_CHK(ids + last, 4)) prev_state[slot] = ids[last];
                }
                if (prev >= 0) row = (int)(((long long)prev * mul_prev + (long long)id * mul_cur) % (long long)buckets);
            }
        }
        s_row = row;
    }
    __syncthreads();
    const TW* er = table + (size_t)id * H;
    float* o = out + (size_t)t * H;
    if (!ZLM_CHK(er, (size_t)H * sizeof(TW))) return;
    if (pair != nullptr) {
        const TW* pr = pair + (size_t)s_row * H;
        if (!ZLM_CHK(pr, (size_t)H * sizeof(TW))) return;
        for (int i = threadIdx.x; i < H; i += blockDim.x) o[i] = fmaf(to_f32(er[i]), scale, to_f32(pr[i]));
    } else {
        for (int i = threadIdx.x; i < H; i += blockDim.x) o[i] = to_f32(er[i]) * scale;
    }
}

extern "C" int zlm_embed_scaled(float* out, const void* table, int dtype, float scale, const void* pair, int buckets,
                                long long mul_prev, long long mul_cur, const int* ids, const int* token_pos,
                                const int* token_seq, const int* cu_seqlens, const int* seq_slot, int* prev_state, int T,
                                int H, int V, cudaStream_t st) {
    if (T == 0) return ZLM_OK;
    ZLM_REQUIRE(T > 0 && H > 0 && V > 0, "embed_scaled: bad sizes T=%d H=%d V=%d", T, H, V);
    ZLM_REQUIRE(pair == nullptr || (buckets > 0 && mul_prev >= 0 && mul_cur >= 0 && token_pos && token_seq && cu_seqlens &&
                                    seq_slot && prev_state),
                "embed_scaled: the pair table needs buckets > 0, multipliers >= 0, the step's arrays and the slots' state");
    const int threads = H >= 1024 ? 256 : 128;
    if (dtype == ZLM_DTYPE_F32)
        zlm_launch(embed_scaled_kernel<float>, T, threads, 0, st, out, (const float*)table, scale, (const float*)pair, buckets,
                   mul_prev, mul_cur, ids, token_pos, token_seq, cu_seqlens, seq_slot, prev_state, H, V);
    else if (dtype == ZLM_DTYPE_BF16)
        zlm_launch(embed_scaled_kernel<__nv_bfloat16>, T, threads, 0, st, out, (const __nv_bfloat16*)table, scale,
                   (const __nv_bfloat16*)pair, buckets, mul_prev, mul_cur, ids, token_pos, token_seq, cu_seqlens, seq_slot,
                   prev_state, H, V);
    else
        ZLM_REQUIRE(false, "embed_scaled: unsupported table dtype %d", dtype);
    return zlm_check_launch("embed_scaled");
}

// ---------------------------------------------------------------- norm of a sublayer's output, scale, residual add
// One block per row; the block's size is a function of H alone, so the order of the sum of squares never depends on
// the batch.  With H a multiple of 4 and up to 4 float4 a thread the row is read once.  `cast_out` (may be null)
// receives the stream's new row rounded to bfloat16: what the next sublayer's products read.
template <typename TY>
__global__ void norm_scale_add_kernel(float* __restrict__ stream, const TY* __restrict__ y, VecW w, VecW ls, int has_ls,
                                      int H, float eps, __nv_bfloat16* __restrict__ cast_out) {
    __shared__ float red[32];
    pdl_trigger();
    const int r = blockIdx.x;
    pdl_wait();
    float* xr = stream + (size_t)r * H;
    const TY* yr = y + (size_t)r * H;
    if (!ZLM_CHK(xr, (size_t)H * 4) || !ZLM_CHK(yr, (size_t)H * sizeof(TY)) ||
        !ZLM_CHK(w.p, (size_t)H * (w.dtype == ZLM_DTYPE_F32 ? 4 : 2)) ||
        (has_ls && !ZLM_CHK(ls.p, (size_t)H * (ls.dtype == ZLM_DTYPE_F32 ? 4 : 2))) ||
        (cast_out && !ZLM_CHK(cast_out + (size_t)r * H, (size_t)H * 2)))
        return;
    __nv_bfloat16* cr = cast_out ? cast_out + (size_t)r * H : nullptr;
    const int nv = H / 4;
    const bool in_regs = sizeof(TY) == 4 && H % 4 == 0 && nv <= NORM_MAX_V4 * (int)blockDim.x;
    float4 v[NORM_MAX_V4];
    float s = 0.f;
    if (in_regs) {
#pragma unroll
        for (int j = 0; j < NORM_MAX_V4; ++j) {
            const int c = threadIdx.x + j * blockDim.x;
            v[j] = c < nv ? *(const float4*)((const float*)yr + c * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
            s = fmaf(v[j].x, v[j].x, s); s = fmaf(v[j].y, v[j].y, s);
            s = fmaf(v[j].z, v[j].z, s); s = fmaf(v[j].w, v[j].w, s);
        }
    } else {
        for (int i = threadIdx.x; i < H; i += blockDim.x) {
            const float a = to_f32(yr[i]);
            s = fmaf(a, a, s);
        }
    }
    const float tot = block_sum(s, red);
    const float inv = 1.0f / sqrtf(tot / (float)H + eps);
    if (in_regs) {
#pragma unroll
        for (int j = 0; j < NORM_MAX_V4; ++j) {
            const int c = threadIdx.x + j * blockDim.x;
            if (c >= nv) continue;
            const int i = c * 4;
            float4 wv = w.load4(i);
            if (has_ls) {
                const float4 l = ls.load4(i);
                // (y * inv * w) * ls, in that order, as two roundings of the norm's result
                float4 a = *(float4*)(xr + i);
                a.x += ((v[j].x * inv) * wv.x) * l.x; a.y += ((v[j].y * inv) * wv.y) * l.y;
                a.z += ((v[j].z * inv) * wv.z) * l.z; a.w += ((v[j].w * inv) * wv.w) * l.w;
                *(float4*)(xr + i) = a;
                if (cr) store4(cr + i, a.x, a.y, a.z, a.w);
            } else {
                float4 a = *(float4*)(xr + i);
                a.x += (v[j].x * inv) * wv.x; a.y += (v[j].y * inv) * wv.y;
                a.z += (v[j].z * inv) * wv.z; a.w += (v[j].w * inv) * wv.w;
                *(float4*)(xr + i) = a;
                if (cr) store4(cr + i, a.x, a.y, a.z, a.w);
            }
        }
    } else {
        for (int i = threadIdx.x; i < H; i += blockDim.x) {
            float n = (to_f32(yr[i]) * inv) * w[i];
            if (has_ls) n *= ls[i];
            const float a = xr[i] + n;
            xr[i] = a;
            if (cr) cr[i] = __float2bfloat16_rn(a);
        }
    }
}

extern "C" int zlm_norm_scale_add(float* stream, const void* y, int y_dtype, const void* w, int w_dtype, const void* ls,
                                  int ls_dtype, int R, int H, float eps, void* cast_out, cudaStream_t st) {
    if (R == 0) return ZLM_OK;
    ZLM_REQUIRE(R > 0 && H > 0, "norm_scale_add: bad sizes R=%d H=%d", R, H);
    ZLM_REQUIRE(H % 4 != 0 || (uintptr_t)cast_out % 8 == 0, "norm_scale_add: the bfloat16 copy must be 8-byte aligned");
    ZLM_REQUIRE(H % 4 != 0 || ((uintptr_t)stream % 16 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)w % 16 == 0 &&
                               (uintptr_t)ls % 16 == 0),
                "norm_scale_add: stream, input and vectors must be 16-byte aligned");
    int threads = 128;
    while (threads < 1024 && threads * 4 * NORM_MAX_V4 < H) threads *= 2;
    VecW vw{w, w_dtype}, vl{ls ? ls : w, ls ? ls_dtype : w_dtype};
    if (y_dtype == ZLM_DTYPE_F32)
        zlm_launch(norm_scale_add_kernel<float>, R, threads, 0, st, stream, (const float*)y, vw, vl, ls ? 1 : 0, H, eps,
                   (__nv_bfloat16*)cast_out);
    else if (y_dtype == ZLM_DTYPE_BF16)
        zlm_launch(norm_scale_add_kernel<__nv_bfloat16>, R, threads, 0, st, stream, (const __nv_bfloat16*)y, vw, vl,
                   ls ? 1 : 0, H, eps, (__nv_bfloat16*)cast_out);
    else
        ZLM_REQUIRE(false, "norm_scale_add: unsupported input dtype %d", y_dtype);
    return zlm_check_launch("norm_scale_add");
}

// ---------------------------------------------------------------- the same, and the norm that reads the stream next
// stream += y / rms(y) * w1, then out2 = norm(stream) * w2 in the element type: a layer that norms a sublayer's
// output and the next sublayer's input does both in one pass over the row, which is held in registers (or, where it does
// not fit them, in shared memory) as fp32.  norm is x / rms(x), or with CENTER d / rms(d), d = x - mean(x) (layer norm).
// One block per row, its size a function of H and of whether the rows are few.
//
// `tail` (steps of one token a sequence; taps 0: none): the next layer's causal convolution over time of the rows just
// normed, mixed[r] = h + sum_j w[j] * u_j with u the taps - 1 rows before (the slot's state, oldest first) and h itself
// last; the state then takes h in.  h is the row as out2 holds it.
#define NAN_FEW_ROWS 128
struct ConvTail {
    const void* w;              // [taps][H] in the element type
    int taps;
    void* state;                // [slots][taps - 1][H] in the element type
    const int* seq_slot;
    void* mixed;                // [rows][H]
};
template <typename TO>
__device__ __forceinline__ float conv_tail_channel(const TO* w, TO* st, int taps, int H, int i, TO hr) {
    float a = 0.f;
    for (int j = 0; j < taps - 1; ++j) {
        const TO u = st[(size_t)j * H + i];
        a = fmaf(to_f32(w[(size_t)j * H + i]), to_f32(u), a);
        if (j > 0) st[(size_t)(j - 1) * H + i] = u;
    }
    if (taps > 1) st[(size_t)(taps - 2) * H + i] = hr;
    const float h = to_f32(hr);
    return h + fmaf(to_f32(w[(size_t)(taps - 1) * H + i]), h, a);
}
// the same for four neighbouring channels
__device__ __forceinline__ float4 tail_load4(const float* p) { return *(const float4*)p; }
__device__ __forceinline__ float4 tail_load4(const __nv_bfloat16* p) {
    const uint2 u = *(const uint2*)p;
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                       __uint_as_float(u.y & 0xffff0000u));
}
template <typename TO>
__device__ __forceinline__ void conv_tail_channels4(const TO* w, TO* st, TO* mixed, int taps, int H, int i, float4 h) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int j = 0; j < taps - 1; ++j) {
        const float4 u = tail_load4(st + (size_t)j * H + i), k = tail_load4(w + (size_t)j * H + i);
        a.x = fmaf(k.x, u.x, a.x); a.y = fmaf(k.y, u.y, a.y); a.z = fmaf(k.z, u.z, a.z); a.w = fmaf(k.w, u.w, a.w);
        if (j > 0) store4(st + (size_t)(j - 1) * H + i, u.x, u.y, u.z, u.w);
    }
    if (taps > 1) store4(st + (size_t)(taps - 2) * H + i, h.x, h.y, h.z, h.w);
    const float4 k = tail_load4(w + (size_t)(taps - 1) * H + i);
    store4(mixed + i, h.x + fmaf(k.x, h.x, a.x), h.y + fmaf(k.y, h.y, a.y), h.z + fmaf(k.z, h.z, a.z), h.w + fmaf(k.w, h.w, a.w));
}
template <typename TO> __device__ __forceinline__ float4 as_stored(float4 v) {
    return make_float4(to_f32(from_f32<TO>(v.x)), to_f32(from_f32<TO>(v.y)), to_f32(from_f32<TO>(v.z)), to_f32(from_f32<TO>(v.w)));
}

// NV: float4s of a row a thread keeps (0: the row in shared memory).  TAPS > 0 (with NV 1): that many taps, whose weights
// and rows of state are asked for at the start, together with the row; TAPS 0: tail.taps of them, one after the other.
template <typename TO, bool CENTER, int NV, int TAPS>
__global__ void __launch_bounds__(1024)
norm_add_norm_kernel(float* __restrict__ stream, const float* __restrict__ y, VecW w1, float eps1,
                                     TO* __restrict__ out2, VecW w2, float eps2, int H, ConvTail tail) {
    extern __shared__ float nan_row[];          // [32] reduction, then (rows that do not fit the registers) [H] the row
    float* red = nan_row;
    float* row = nan_row + 32;
    pdl_trigger();
    const int r = blockIdx.x;
    const TO* cw = (const TO*)tail.w;
    float4 k1[NV > 0 ? NV : 1], k2[NV > 0 ? NV : 1], ck[TAPS > 0 ? TAPS : 1], cu[TAPS > 1 ? TAPS - 1 : 1];
    if (NV == 1) {
        // few rows: what does not change during a step is asked for ahead of the wait
        if ((int)threadIdx.x * 4 < H) {
            k1[0] = w1.load4(threadIdx.x * 4);
            k2[0] = w2.load4(threadIdx.x * 4);
            if (TAPS > 0 && ZLM_CHK(cw, (size_t)TAPS * H * sizeof(TO)))
#pragma unroll
                for (int j = 0; j < TAPS; ++j) ck[j] = tail_load4(cw + (size_t)j * H + threadIdx.x * 4);
        }
    }
    pdl_wait();
    float* xr = stream + (size_t)r * H;
    const float* yr = y + (size_t)r * H;
    TO* orow = out2 + (size_t)r * H;
    if (!ZLM_CHK(xr, (size_t)H * 4) || !ZLM_CHK(yr, (size_t)H * 4) || !ZLM_CHK(orow, (size_t)H * sizeof(TO))) return;
    TO *st = nullptr, *mixed = nullptr;
    if (tail.taps > 0) {
        if (!ZLM_CHK(tail.seq_slot + r, 4)) return;
        mixed = (TO*)tail.mixed + (size_t)r * H;
        if (tail.taps > 1) st = (TO*)tail.state + (size_t)tail.seq_slot[r] * (tail.taps - 1) * H;
        if (!ZLM_CHK(mixed, (size_t)H * sizeof(TO)) || !ZLM_CHK(cw, (size_t)tail.taps * H * sizeof(TO)) ||
            (st && !ZLM_CHK(st, (size_t)(tail.taps - 1) * H * sizeof(TO))))
            return;
    }
    if (NV > 0) {
        // H a multiple of 4 and up to NV float4 a thread: the row is read once and stays in registers
        const int nv = H / 4;
        float4 v[NV > 0 ? NV : 1], x[NV > 0 ? NV : 1];
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int c = threadIdx.x + j * blockDim.x;
            v[j] = c < nv ? *(const float4*)(yr + c * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
            x[j] = c < nv ? *(const float4*)(xr + c * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        if (TAPS > 1 && (int)threadIdx.x < nv)
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) cu[j] = tail_load4(st + (size_t)j * H + threadIdx.x * 4);
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            s = fmaf(v[j].x, v[j].x, s); s = fmaf(v[j].y, v[j].y, s);
            s = fmaf(v[j].z, v[j].z, s); s = fmaf(v[j].w, v[j].w, s);
        }
        const float inv1 = 1.0f / sqrtf(block_sum(s, red) / (float)H + eps1);
        float s2 = 0.f;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int c = threadIdx.x + j * blockDim.x;
            if (c >= nv) continue;
            const float4 wv = NV == 1 ? k1[0] : w1.load4(c * 4);
            float4 a = x[j];
            a.x += (v[j].x * inv1) * wv.x; a.y += (v[j].y * inv1) * wv.y;
            a.z += (v[j].z * inv1) * wv.z; a.w += (v[j].w * inv1) * wv.w;
            *(float4*)(xr + c * 4) = a;
            v[j] = a;
            if (CENTER) {
                s2 += (a.x + a.y) + (a.z + a.w);
            } else {
                s2 = fmaf(a.x, a.x, s2); s2 = fmaf(a.y, a.y, s2); s2 = fmaf(a.z, a.z, s2); s2 = fmaf(a.w, a.w, s2);
            }
        }
        float sq = block_sum(s2, red);
        if (CENTER) {
            const float mean = sq / (float)H;
            float q = 0.f;
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                if ((int)(threadIdx.x + j * blockDim.x) >= nv) continue;
                v[j].x -= mean; v[j].y -= mean; v[j].z -= mean; v[j].w -= mean;
                q = fmaf(v[j].x, v[j].x, q); q = fmaf(v[j].y, v[j].y, q); q = fmaf(v[j].z, v[j].z, q); q = fmaf(v[j].w, v[j].w, q);
            }
            sq = block_sum(q, red);
        }
        const float inv2 = 1.0f / sqrtf(sq / (float)H + eps2);
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int c = threadIdx.x + j * blockDim.x;
            if (c >= nv) continue;
            const float4 wv = NV == 1 ? k2[0] : w2.load4(c * 4);
            const float4 h = make_float4((v[j].x * inv2) * wv.x, (v[j].y * inv2) * wv.y, (v[j].z * inv2) * wv.z, (v[j].w * inv2) * wv.w);
            store4(orow + c * 4, h.x, h.y, h.z, h.w);
            if (TAPS > 0) {
                const float4 hs = as_stored<TO>(h);
                float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int t = 0; t < TAPS; ++t) {
                    const float4 u = t < TAPS - 1 ? cu[t < TAPS - 1 ? t : 0] : hs;
                    a.x = fmaf(ck[t].x, u.x, a.x); a.y = fmaf(ck[t].y, u.y, a.y);
                    a.z = fmaf(ck[t].z, u.z, a.z); a.w = fmaf(ck[t].w, u.w, a.w);
                    if (t > 0) store4(st + (size_t)(t - 1) * H + c * 4, u.x, u.y, u.z, u.w);
                }
                store4(mixed + c * 4, hs.x + a.x, hs.y + a.y, hs.z + a.z, hs.w + a.w);
            } else if (tail.taps > 0) {
                conv_tail_channels4<TO>(cw, st, mixed, tail.taps, H, c * 4, as_stored<TO>(h));
            }
        }
        return;
    }
    float s = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float a = yr[i];
        row[i] = a;
        s = fmaf(a, a, s);
    }
    const float inv1 = 1.0f / sqrtf(block_sum(s, red) / (float)H + eps1);
    float s2 = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float a = xr[i] + (row[i] * inv1) * w1[i];
        xr[i] = a;
        row[i] = a;
        s2 = CENTER ? s2 + a : fmaf(a, a, s2);
    }
    float sq = block_sum(s2, red), mean = 0.f;
    if (CENTER) {
        mean = sq / (float)H;
        float q = 0.f;
        for (int i = threadIdx.x; i < H; i += blockDim.x) {
            const float d = row[i] - mean;
            q = fmaf(d, d, q);
        }
        sq = block_sum(q, red);
    }
    const float inv2 = 1.0f / sqrtf(sq / (float)H + eps2);
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const TO h = from_f32<TO>(((row[i] - mean) * inv2) * w2[i]);
        orow[i] = h;
        if (tail.taps > 0) mixed[i] = from_f32<TO>(conv_tail_channel<TO>(cw, st, tail.taps, H, i, h));
    }
}

template <typename TO, bool CENTER>
static void launch_norm_add_norm(int R, cudaStream_t st, float* stream, const float* y, VecW v1, float eps1, void* out2, VecW v2,
                                 float eps2, int H, bool even, ConvTail tail) {
    int threads = 128;
    if (even && R <= NAN_FEW_ROWS && H <= 4096) {
        // few rows: the whole latency of one row counts, so a thread has one float4 of it
        while (threads * 4 < H) threads *= 2;
#define ZLM_NAN(TAPS)                                                                                                        \
        zlm_launch(norm_add_norm_kernel<TO, CENTER, 1, TAPS>, R, threads, 32 * sizeof(float), st, stream, y, v1, eps1, (TO*)out2, v2, \
                   eps2, H, tail)
        if (tail.taps == 2) ZLM_NAN(2);
        else if (tail.taps == 3) ZLM_NAN(3);
        else if (tail.taps == 4) ZLM_NAN(4);
        else ZLM_NAN(0);
#undef ZLM_NAN
        return;
    }
    while (threads < 1024 && threads * 4 * NORM_MAX_V4 < H) threads *= 2;
    if (even && H <= threads * 4 * NORM_MAX_V4)
        zlm_launch(norm_add_norm_kernel<TO, CENTER, NORM_MAX_V4, 0>, R, threads, 32 * sizeof(float), st, stream, y, v1, eps1, (TO*)out2,
                   v2, eps2, H, tail);
    else
        zlm_launch(norm_add_norm_kernel<TO, CENTER, 0, 0>, R, threads, (32 + (size_t)H) * sizeof(float), st, stream, y, v1, eps1,
                   (TO*)out2, v2, eps2, H, tail);
}

// center 1: the second norm is a layer norm.  taps 0: no convolution (conv_w, state, seq_slot and mixed are not used).
extern "C" int zlm_norm_add_norm(float* stream, const float* y, const void* w1, int w1_dtype, float eps1, void* out2,
                                 int out2_dtype, const void* w2, int w2_dtype, float eps2, int R, int H, int center,
                                 const void* conv_w, int taps, void* state, const int* seq_slot, void* mixed, cudaStream_t st) {
    if (R == 0) return ZLM_OK;
    ZLM_REQUIRE(R > 0 && H > 0 && H <= 11264, "norm_add_norm: bad sizes R=%d H=%d (rows of up to 11264)", R, H);
    ZLM_REQUIRE(taps >= 0 && (taps == 0 || (conv_w && mixed && seq_slot && (taps == 1 || state))),
                "norm_add_norm: a convolution of %d taps needs its weights, the slots' state and a place for its rows", taps);
    const bool even = H % 4 == 0 && (uintptr_t)stream % 16 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)w1 % 16 == 0 &&
                      (uintptr_t)w2 % 16 == 0 && (uintptr_t)out2 % 16 == 0 && (uintptr_t)conv_w % 16 == 0 &&
                      (uintptr_t)state % 16 == 0 && (uintptr_t)mixed % 16 == 0;
    const VecW v1{w1, w1_dtype}, v2{w2, w2_dtype};
    const ConvTail tail{conv_w, taps, state, seq_slot, mixed};
#define ZLM_NAN(TO)                                                                                                     \
    do {                                                                                                                \
        if (center) launch_norm_add_norm<TO, true>(R, st, stream, y, v1, eps1, out2, v2, eps2, H, even, tail);           \
        else launch_norm_add_norm<TO, false>(R, st, stream, y, v1, eps1, out2, v2, eps2, H, even, tail);                 \
    } while (0)
    if (out2_dtype == ZLM_DTYPE_F32) ZLM_NAN(float);
    else if (out2_dtype == ZLM_DTYPE_BF16) ZLM_NAN(__nv_bfloat16);
    else ZLM_REQUIRE(false, "norm_add_norm: unsupported output dtype %d", out2_dtype);
#undef ZLM_NAN
    return zlm_check_launch("norm_add_norm");
}

// ---------------------------------------------------------------- a polynomial of normed powers
// out[t] = a N(z) + b N(z^2) + c N(z^3) + e over the row z[t] of ff values (powers element by element, N(u) = u /
// sqrt(mean(u^2) + eps)), the four numbers in `coef`; columns of out from ff up to out_cols become zeros.  Sums and
// norms fp32.  One block per row, its size a function of ff alone.
#define PN_MAX_V 4
template <typename TA> struct PolyVec;          // eight neighbouring elements
template <> struct PolyVec<__nv_bfloat16> {
    uint4 u;
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { u = *(const uint4*)p; }
    __device__ __forceinline__ float get(int i) const {
        const unsigned w = i < 2 ? u.x : (i < 4 ? u.y : (i < 6 ? u.z : u.w));
        return __uint_as_float((i & 1) ? (w & 0xffff0000u) : (w << 16));
    }
};
template <> struct PolyVec<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) { a = *(const float4*)p; b = *(const float4*)(p + 4); }
    __device__ __forceinline__ float get(int i) const {
        const float4 v = i < 4 ? a : b;
        const int k = i & 3;
        return k == 0 ? v.x : (k == 1 ? v.y : (k == 2 ? v.z : v.w));
    }
};
template <typename TA>
__global__ void poly_norm_kernel(TA* __restrict__ out, int out_stride, int out_cols, const TA* __restrict__ z, int z_stride,
                                 VecW coef, int F, float eps, int in_regs) {
    __shared__ float red[32];
    pdl_trigger();
    const int t = blockIdx.x;
    pdl_wait();
    const TA* zr = z + (size_t)t * z_stride;
    TA* o = out + (size_t)t * out_stride;
    if (!ZLM_CHK(zr, (size_t)F * sizeof(TA)) || !ZLM_CHK(o, (size_t)out_cols * sizeof(TA)) ||
        !ZLM_CHK(coef.p, 4 * (coef.dtype == ZLM_DTYPE_F32 ? 4 : 2)))
        return;
    float s1 = 0.f, s2 = 0.f, s3 = 0.f;
    auto add = [&](float v) {
        const float q = v * v;
        s1 += q;
        s2 = fmaf(q, q, s2);
        s3 = fmaf(q * q, q, s3);
    };
    PolyVec<TA> keep[PN_MAX_V];
    const int nv = F / 8;
    if (in_regs) {
#pragma unroll
        for (int j = 0; j < PN_MAX_V; ++j) {
            const int c = threadIdx.x + j * blockDim.x;
            if (c < nv) keep[j].load(zr + c * 8);
        }
#pragma unroll
        for (int j = 0; j < PN_MAX_V; ++j) {
            if (threadIdx.x + j * blockDim.x >= nv) continue;
#pragma unroll
            for (int i = 0; i < 8; ++i) add(keep[j].get(i));
        }
    } else {
        for (int i = threadIdx.x; i < F; i += blockDim.x) add(to_f32(zr[i]));
    }
    const float f = (float)F;
    const float ka = coef[0] / sqrtf(block_sum(s1, red) / f + eps);
    const float kb = coef[1] / sqrtf(block_sum(s2, red) / f + eps);
    const float kc = coef[2] / sqrtf(block_sum(s3, red) / f + eps);
    const float ke = coef[3];
    auto value = [&](float v) { return fmaf(v, fmaf(v, fmaf(v, kc, kb), ka), ke); };
    if (in_regs) {
#pragma unroll
        for (int j = 0; j < PN_MAX_V; ++j) {
            const int c = threadIdx.x + j * blockDim.x;
            if (c >= nv) continue;
            store4(o + c * 8, value(keep[j].get(0)), value(keep[j].get(1)), value(keep[j].get(2)), value(keep[j].get(3)));
            store4(o + c * 8 + 4, value(keep[j].get(4)), value(keep[j].get(5)), value(keep[j].get(6)), value(keep[j].get(7)));
        }
    } else {
        for (int i = threadIdx.x; i < F; i += blockDim.x) o[i] = from_f32<TA>(value(to_f32(zr[i])));
    }
    for (int i = F + threadIdx.x; i < out_cols; i += blockDim.x) o[i] = from_f32<TA>(0.f);
}

extern "C" int zlm_poly_norm(void* out, int out_stride, int out_cols, const void* z, int z_stride, int dtype, const void* coef,
                             int coef_dtype, int T, int F, float eps, cudaStream_t st) {
    if (T == 0) return ZLM_OK;
    ZLM_REQUIRE(T > 0 && F > 0 && out_cols >= F && out_stride >= out_cols && z_stride >= F, "poly_norm: bad sizes T=%d F=%d", T, F);
    int threads = 128;
    while (threads < 1024 && threads * 8 * PN_MAX_V < F) threads *= 2;
    const int el = dtype == ZLM_DTYPE_F32 ? 4 : 2;
    const int in_regs = (F % 8 == 0 && F <= threads * 8 * PN_MAX_V && ((size_t)z_stride * el) % 16 == 0 &&
                         ((size_t)out_stride * el) % 16 == 0 && (uintptr_t)z % 16 == 0 && (uintptr_t)out % 16 == 0) ? 1 : 0;
    const VecW c{coef, coef_dtype};
    if (dtype == ZLM_DTYPE_F32)
        zlm_launch(poly_norm_kernel<float>, T, threads, 0, st, (float*)out, out_stride, out_cols, (const float*)z, z_stride, c, F,
                   eps, in_regs);
    else if (dtype == ZLM_DTYPE_BF16)
        zlm_launch(poly_norm_kernel<__nv_bfloat16>, T, threads, 0, st, (__nv_bfloat16*)out, out_stride, out_cols,
                   (const __nv_bfloat16*)z, z_stride, c, F, eps, in_regs);
    else
        ZLM_REQUIRE(false, "poly_norm: unsupported dtype %d", dtype);
    return zlm_check_launch("poly_norm");
}

// ---------------------------------------------------------------- the stream's rows in the compute dtype
__global__ void cast_rows_kernel(__nv_bfloat16* __restrict__ out, const float* __restrict__ x, size_t n4, size_t n) {
    pdl_launch_dependents();
    pdl_wait();
    for (size_t c = (size_t)blockIdx.x * blockDim.x + threadIdx.x; c < n4; c += (size_t)gridDim.x * blockDim.x) {
        if (!ZLM_CHK(x + c * 4, 16) || !ZLM_CHK(out + c * 4, 8)) continue;
        const float4 v = *(const float4*)(x + c * 4);
        store4(out + c * 4, v.x, v.y, v.z, v.w);
    }
    // a tail of up to three elements
    if (blockIdx.x == 0)
        for (size_t i = n4 * 4 + threadIdx.x; i < n; i += blockDim.x)
            if (ZLM_CHK(x + i, 4) && ZLM_CHK(out + i, 2)) out[i] = __float2bfloat16_rn(x[i]);
}

extern "C" int zlm_cast_rows(void* out, const float* x, long long n, cudaStream_t st) {
    if (n == 0) return ZLM_OK;
    ZLM_REQUIRE(n > 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)out % 8 == 0, "cast_rows: %lld elements, aligned operands", n);
    const size_t n4 = (size_t)n / 4;
    long long blocks = (long long)((n4 + 255) / 256);
    if (blocks < 1) blocks = 1;
    if (blocks > 148 * 8) blocks = 148 * 8;
    zlm_launch(cast_rows_kernel, (int)blocks, 256, 0, st, (__nv_bfloat16*)out, x, n4, (size_t)n);
    return zlm_check_launch("cast_rows");
}

// ---------------------------------------------------------------- gated activation
__device__ __forceinline__ float zlm_gelu_tanh(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// gu is [T, 2I]: gate in columns [0, I), up in [I, 2I); act 0: silu, 1: the tanh form of gelu
template <typename TA>
__global__ void gated_act_kernel(TA* __restrict__ out, const TA* __restrict__ gu, int T, int I, int act) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t n = (size_t)T * I;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < n; e += (size_t)gridDim.x * blockDim.x) {
        const size_t t = e / I;
        const int i = (int)(e - t * I);
        if (!ZLM_CHK(&gu[t * 2 * I + i], sizeof(TA)) || !ZLM_CHK(&gu[t * 2 * I + I + i], sizeof(TA)) ||
            !ZLM_CHK(&out[e], sizeof(TA)))
            continue;
        const float g = to_f32(gu[t * 2 * I + i]);
        const float u = to_f32(gu[t * 2 * I + I + i]);
        const float a = act == 1 ? zlm_gelu_tanh(g) : g / (1.0f + expf(-g));
        out[e] = from_f32<TA>(a * u);
    }
}

extern "C" int zlm_gated_act(void* out, const void* gu, int dtype, int T, int I, int act, cudaStream_t st) {
    if (T == 0) return ZLM_OK;
    ZLM_REQUIRE(T > 0 && I > 0 && (act == 0 || act == 1), "gated_act: bad sizes T=%d I=%d act=%d", T, I, act);
    const size_t n = (size_t)T * I;
    int blocks = (int)((n + 255) / 256);
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == ZLM_DTYPE_F32)
        zlm_launch(gated_act_kernel<float>, blocks, 256, 0, st, (float*)out, (const float*)gu, T, I, act);
    else if (dtype == ZLM_DTYPE_BF16)
        zlm_launch(gated_act_kernel<__nv_bfloat16>, blocks, 256, 0, st, (__nv_bfloat16*)out, (const __nv_bfloat16*)gu, T, I, act);
    else
        ZLM_REQUIRE(false, "gated_act: unsupported dtype %d", dtype);
    return zlm_check_launch("gated_act");
}

// ---------------------------------------------------------------- x *= s
__global__ void scale_f32_kernel(float* __restrict__ x, size_t n, float s) {
    pdl_launch_dependents();
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        if (ZLM_CHK(x + i, 4)) x[i] *= s;
}

extern "C" int zlm_scale_f32(float* x, long long n, float s, cudaStream_t st) {
    if (n <= 0) return ZLM_OK;
    long long blocks = (n + 255) / 256;
    if (blocks > 148 * 8) blocks = 148 * 8;
    zlm_launch(scale_f32_kernel, (int)blocks, 256, 0, st, x, (size_t)n, s);
    return zlm_check_launch("scale_f32");
}

// ---------------------------------------------------------------- out (+)= alpha a + beta b
// The sum of two sublayers that ran side by side on one input, each with a scale of its own; fp32.
__global__ void scaled_sum_kernel(float* __restrict__ out, const float* __restrict__ a, float alpha, const float* __restrict__ b,
                                  float beta, size_t n, int accumulate) {
    pdl_launch_dependents();
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        if (!ZLM_CHK(out + i, 4) || !ZLM_CHK(a + i, 4) || !ZLM_CHK(b + i, 4)) continue;
        const float y = fmaf(alpha, a[i], beta * b[i]);
        out[i] = accumulate ? out[i] + y : y;
    }
}

extern "C" int zlm_scaled_sum(float* out, const float* a, float alpha, const float* b, float beta, long long n, int accumulate,
                              cudaStream_t st) {
    if (n <= 0) return ZLM_OK;
    long long blocks = (n + 255) / 256;
    if (blocks > 148 * 8) blocks = 148 * 8;
    zlm_launch(scaled_sum_kernel, (int)blocks, 256, 0, st, out, a, alpha, b, beta, (size_t)n, accumulate);
    return zlm_check_launch("scaled_sum");
}

// ---------------------------------------------------------------- x = cap * tanh(x / cap)
__global__ void softcap_f32_kernel(float* __restrict__ x, size_t n, float cap) {
    pdl_launch_dependents();
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        if (ZLM_CHK(x + i, 4)) x[i] = cap * tanhf(x[i] / cap);
}

extern "C" int zlm_softcap_f32(float* x, long long n, float cap, cudaStream_t st) {
    if (n <= 0) return ZLM_OK;
    ZLM_REQUIRE(cap > 0.f, "softcap: cap %g", (double)cap);
    long long blocks = (n + 255) / 256;
    if (blocks > 148 * 8) blocks = 148 * 8;
    zlm_launch(softcap_f32_kernel, (int)blocks, 256, 0, st, x, (size_t)n, cap);
    return zlm_check_launch("softcap_f32");
}

// ---------------------------------------------------------------- silu in place on the first columns of every row
template <typename TA>
__global__ void silu_rows_kernel(TA* __restrict__ x, int stride, int T, int cols) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t n = (size_t)T * cols;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < n; e += (size_t)gridDim.x * blockDim.x) {
        const size_t t = e / cols;
        TA* p = x + t * stride + (e - t * cols);
        if (!ZLM_CHK(p, sizeof(TA))) continue;
        const float z = to_f32(*p);
        *p = from_f32<TA>(z / (1.0f + expf(-z)));
    }
}

extern "C" int zlm_silu_rows(void* x, int stride, int dtype, int T, int cols, cudaStream_t st) {
    if (T <= 0 || cols <= 0) return ZLM_OK;
    ZLM_REQUIRE(stride >= cols, "silu_rows: %d columns in rows of %d", cols, stride);
    const size_t n = (size_t)T * cols;
    int blocks = (int)((n + 255) / 256 > 148 * 16 ? 148 * 16 : (n + 255) / 256);
    if (dtype == ZLM_DTYPE_F32)
        zlm_launch(silu_rows_kernel<float>, blocks, 256, 0, st, (float*)x, stride, T, cols);
    else if (dtype == ZLM_DTYPE_BF16)
        zlm_launch(silu_rows_kernel<__nv_bfloat16>, blocks, 256, 0, st, (__nv_bfloat16*)x, stride, T, cols);
    else
        ZLM_REQUIRE(false, "silu_rows: unsupported dtype %d", dtype);
    return zlm_check_launch("silu_rows");
}

// ---------------------------------------------------------------- gated activation with clamped operands
// out = g' * sigmoid(alpha g') * (u' + 1), g' = min(gate, limit), u' = clamp(up, -limit, limit); gu is [T, 2I]: gate in
// columns [0, I), up in [I, 2I)
template <typename TA>
__global__ void gated_limit_kernel(TA* __restrict__ out, const TA* __restrict__ gu, int T, int I, float limit, float alpha) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t n = (size_t)T * I;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < n; e += (size_t)gridDim.x * blockDim.x) {
        const size_t t = e / I;
        const int i = (int)(e - t * I);
        if (!ZLM_CHK(&gu[t * 2 * I + i], sizeof(TA)) || !ZLM_CHK(&gu[t * 2 * I + I + i], sizeof(TA)) ||
            !ZLM_CHK(&out[e], sizeof(TA)))
            continue;
        const float g = fminf(to_f32(gu[t * 2 * I + i]), limit);
        const float u = fminf(fmaxf(to_f32(gu[t * 2 * I + I + i]), -limit), limit);
        out[e] = from_f32<TA>(g / (1.0f + expf(-alpha * g)) * (u + 1.0f));
    }
}

extern "C" int zlm_gated_limit(void* out, const void* gu, int dtype, int T, int I, float limit, float alpha, cudaStream_t st) {
    if (T == 0) return ZLM_OK;
    ZLM_REQUIRE(T > 0 && I > 0 && limit > 0.f, "gated_limit: bad sizes T=%d I=%d limit=%g", T, I, (double)limit);
    const size_t n = (size_t)T * I;
    int blocks = (int)((n + 255) / 256);
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == ZLM_DTYPE_F32)
        zlm_launch(gated_limit_kernel<float>, blocks, 256, 0, st, (float*)out, (const float*)gu, T, I, limit, alpha);
    else if (dtype == ZLM_DTYPE_BF16)
        zlm_launch(gated_limit_kernel<__nv_bfloat16>, blocks, 256, 0, st, (__nv_bfloat16*)out, (const __nv_bfloat16*)gu, T, I,
                   limit, alpha);
    else
        ZLM_REQUIRE(false, "gated_limit: unsupported dtype %d", dtype);
    return zlm_check_launch("gated_limit");
}

// ---------------------------------------------------------------- one gate number per head
// x [T, heads, V] (any token and head strides) *= sigmoid(g[t, h]); a warp per (token, head)
template <typename TA>
__global__ void head_scalar_gate_kernel(TA* __restrict__ x, int x_stride, int x_hstride, const TA* __restrict__ g,
                                        int g_stride, int T, int H, int V) {
    pdl_trigger();
    const int lane = threadIdx.x & 31;
    const long long unit = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (unit >= (long long)T * H) return;
    const int t = (int)(unit / H), h = (int)(unit % H);
    pdl_wait();
    TA* xp = x + (size_t)t * x_stride + (size_t)h * x_hstride;
    const TA* gp = g + (size_t)t * g_stride + h;
    if (!ZLM_CHK(xp, (size_t)V * sizeof(TA)) || !ZLM_CHK(gp, sizeof(TA))) return;
    const float gate = 1.0f / (1.0f + expf(-to_f32(*gp)));
    for (int e = lane; e < V; e += 32) xp[e] = from_f32<TA>(to_f32(xp[e]) * gate);
}

extern "C" int zlm_head_scalar_gate(void* x, int x_stride, int x_hstride, const void* g, int g_stride, int dtype, int T,
                                    int H, int V, cudaStream_t st) {
    if (T == 0) return ZLM_OK;
    ZLM_REQUIRE(H > 0 && V > 0, "head_scalar_gate: %d heads of %d", H, V);
    const long long units = (long long)T * H;
    const int blocks = (int)((units + 3) / 4);
    if (dtype == ZLM_DTYPE_F32)
        zlm_launch(head_scalar_gate_kernel<float>, blocks, 128, 0, st, (float*)x, x_stride, x_hstride, (const float*)g,
                   g_stride, T, H, V);
    else if (dtype == ZLM_DTYPE_BF16)
        zlm_launch(head_scalar_gate_kernel<__nv_bfloat16>, blocks, 128, 0, st, (__nv_bfloat16*)x, x_stride, x_hstride,
                   (const __nv_bfloat16*)g, g_stride, T, H, V);
    else
        ZLM_REQUIRE(false, "head_scalar_gate: unsupported dtype %d", dtype);
    return zlm_check_launch("head_scalar_gate");
}

ZLM_TRANSLATION_UNIT(stream_ops)
