// Layer norm with a gain and no bias, alone and fused with the residual sum ahead of it:
//
//     n(x) = (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * w
//     layernorm:            out[r] = n(x[rows[r] or r])
//     residual_layernorm:   h += post ? y / sqrt(mean(y^2) + eps_post) * (off_post + w_post) : y;   out = n(h)
//
// y may come as n_parts partial sums, part_stride elements apart, which are added in order while loading.  One block
// per row; the variance is the mean of the squared deviations (a second sum over the row, which the block holds in
// registers: no second trip to memory).  All arithmetic is float, the result is rounded once.
#include "common.cuh"

namespace {

__device__ __forceinline__ void load4(const float* p, float (&v)[4]) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
}
__device__ __forceinline__ void load4(const bf16* p, float (&v)[4]) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
__device__ __forceinline__ void store4(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void store4(bf16* p, const float (&v)[4]) {
    uint2 t;
    *reinterpret_cast<__nv_bfloat162*>(&t.x) = __floats2bfloat162_rn(v[0], v[1]);
    *reinterpret_cast<__nv_bfloat162*>(&t.y) = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = t;
}

struct NormArgs {
    const float* x;            // layernorm: the rows; residual_layernorm: unused
    const int32_t* rows;
    float* h;                  // residual_layernorm: the stream, updated in place (null: layernorm)
    const float* y;
    int n_parts;
    long long part_stride;
    const void* w_post;
    float eps_post, off_post;
    const void* w;
    float eps;
    void* out;
    int hidden;
};

// C > 0: the row in registers, four neighbours a thread and chunk of 1024; C = 0: any width, plain loops.
// ONE: y in one part (a prompt): without the room for several parts' loads more blocks share an SM.
template <typename W, typename O, int C, bool ONE>
__global__ void __launch_bounds__(256, ONE ? (C <= 2 ? 6 : C <= 4 ? 4 : 2) : (C <= 2 ? 4 : C <= 4 ? 3 : 1)) layernorm_kernel(NormArgs a) {
    __shared__ float scratch[64];
    const int r = blockIdx.x, hidden = a.hidden;
    const float inv_n = 1.0f / (float)hidden;
    const W* w = (const W*)a.w;
    const W* wp = (const W*)a.w_post;
    O* dst = (O*)a.out + (size_t)r * hidden;
    float* hr = a.h ? a.h + (size_t)r * hidden : nullptr;
    const float* yr = a.y + (size_t)r * hidden;
    pdl_trigger();
    if constexpr (C == 0) {
        pdl_wait();
        const float* src = hr ? hr : a.x + (size_t)(a.rows ? a.rows[r] : r) * hidden;
        if (hr) {
            auto y_at = [&](int i) {
                float v = yr[i];
                for (int s = 1; s < a.n_parts; ++s) v += yr[(size_t)s * a.part_stride + i];
                return v;
            };
            float inv_post = 1.0f;
            if (wp) {
                float ss = 0.0f;
                for (int i = threadIdx.x; i < hidden; i += blockDim.x) { const float v = y_at(i); ss += v * v; }
                inv_post = rsqrtf(block_sum(ss, scratch) * inv_n + a.eps_post);
            }
            for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
                float v = y_at(i);
                if (wp) v = v * inv_post * (a.off_post + to_float(wp[i]));
                hr[i] += v;
            }
        }
        // every thread reads back only what it wrote itself
        float s = 0.0f;
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) s += src[i];
        const float mean = block_sum(s, scratch) * inv_n;
        float ss = 0.0f;
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) { const float d = src[i] - mean; ss += d * d; }
        const float inv = rsqrtf(block_sum(ss, scratch) * inv_n + a.eps);
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) dst[i] = from_float<O>((src[i] - mean) * inv * to_float(w[i]));
        return;
    } else {
        // the gains are weights: on their way into the L1 while the kernel before this one finishes
        const size_t line = (size_t)threadIdx.x * 128;
        if (line < (size_t)hidden * sizeof(W)) {
            if (wp) prefetch_l1(reinterpret_cast<const char*>(wp) + line);
            prefetch_l1(reinterpret_cast<const char*>(w) + line);
        }
        pdl_wait();
        float res[C][4];
        const float* src = hr ? hr : a.x + (size_t)(a.rows ? a.rows[r] : r) * hidden;
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const int i = (c * 256 + threadIdx.x) * 4;
            res[c][0] = res[c][1] = res[c][2] = res[c][3] = 0.0f;
            if (i < hidden) load4(src + i, res[c]);
        }
        int turn = 0;
        if (hr) {
            float v[C][4];
#pragma unroll
            for (int c = 0; c < C; ++c) {
                const int i = (c * 256 + threadIdx.x) * 4;
                v[c][0] = v[c][1] = v[c][2] = v[c][3] = 0.0f;
                if constexpr (ONE) {
                    if (i < hidden) load4(yr + i, v[c]);
                } else if (i < hidden) {
                    constexpr int AT_ONCE = 4;       // slices whose loads go out together
                    for (int s0 = 0; s0 < a.n_parts; s0 += AT_ONCE) {
                        float t[AT_ONCE][4];
#pragma unroll
                        for (int s = 0; s < AT_ONCE; ++s)
                            if (s0 + s < a.n_parts) load4(yr + (size_t)(s0 + s) * a.part_stride + i, t[s]);
#pragma unroll
                        for (int s = 0; s < AT_ONCE; ++s)
                            if (s0 + s < a.n_parts) {
#pragma unroll
                                for (int e = 0; e < 4; ++e) v[c][e] += t[s][e];
                            }
                    }
                }
            }
            if (wp) {
                float ss = 0.0f;
#pragma unroll
                for (int c = 0; c < C; ++c) ss += v[c][0] * v[c][0] + v[c][1] * v[c][1] + v[c][2] * v[c][2] + v[c][3] * v[c][3];
                const float inv_post = rsqrtf(block_sum_once(ss, scratch, turn) * inv_n + a.eps_post);
                turn ^= 1;
#pragma unroll
                for (int c = 0; c < C; ++c) {
                    const int i = (c * 256 + threadIdx.x) * 4;
                    float g[4] = {0.0f, 0.0f, 0.0f, 0.0f};
                    if (i < hidden) load4(wp + i, g);
#pragma unroll
                    for (int e = 0; e < 4; ++e) v[c][e] = v[c][e] * inv_post * (a.off_post + g[e]);
                }
            }
#pragma unroll
            for (int c = 0; c < C; ++c) {
                const int i = (c * 256 + threadIdx.x) * 4;
#pragma unroll
                for (int e = 0; e < 4; ++e) res[c][e] += v[c][e];
                if (i < hidden) store4(hr + i, res[c]);
            }
        }
        float s = 0.0f;
#pragma unroll
        for (int c = 0; c < C; ++c) s += (res[c][0] + res[c][1]) + (res[c][2] + res[c][3]);
        const float mean = block_sum_once(s, scratch, turn) * inv_n;
        turn ^= 1;
        float ss = 0.0f;
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const bool in = (c * 256 + (int)threadIdx.x) * 4 < hidden;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                res[c][e] = in ? res[c][e] - mean : 0.0f;
                ss += res[c][e] * res[c][e];
            }
        }
        const float inv = rsqrtf(block_sum_once(ss, scratch, turn) * inv_n + a.eps);
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const int i = (c * 256 + threadIdx.x) * 4;
            if (i < hidden) {
                float g[4], o[4];
                load4(w + i, g);
#pragma unroll
                for (int e = 0; e < 4; ++e) o[e] = res[c][e] * inv * g[e];
                store4(dst + i, o);
            }
        }
    }
}

template <typename W, typename O>
int launch_norm(const NormArgs& a, int n, cudaStream_t s) {
    const uintptr_t bits = (uintptr_t)a.x | (uintptr_t)a.h | (uintptr_t)a.y | (uintptr_t)a.w | (uintptr_t)a.w_post |
                           (uintptr_t)a.out;
    int c = 0;
    if (a.hidden % 4 == 0 && !(bits & 15) && a.part_stride % 4 == 0)
        c = a.hidden <= 1024 ? 1 : a.hidden <= 2048 ? 2 : a.hidden <= 3072 ? 3 : a.hidden <= 4096 ? 4 : a.hidden <= 8192 ? 8 : 0;
    const bool one = a.n_parts <= 1;
#define BROLM_LN(C) return one ? launch_pdl(layernorm_kernel<W, O, C, true>, dim3(n), dim3(256), 0, s, a) \
                               : launch_pdl(layernorm_kernel<W, O, C, false>, dim3(n), dim3(256), 0, s, a)
    if (c == 1) BROLM_LN(1);
    if (c == 2) BROLM_LN(2);
    if (c == 3) BROLM_LN(3);
    if (c == 4) BROLM_LN(4);
    if (c == 8) BROLM_LN(8);
#undef BROLM_LN
    return launch_pdl(layernorm_kernel<W, O, 0, false>, dim3(n), dim3(256), 0, s, a);
}

int launch_any(const NormArgs& a, int w_dtype, int out_dtype, int n, cudaStream_t s) {
    if (w_dtype == BROLM_F32 && out_dtype == BROLM_F32) return launch_norm<float, float>(a, n, s);
    if (w_dtype == BROLM_F32 && out_dtype == BROLM_BF16) return launch_norm<float, bf16>(a, n, s);
    if (w_dtype == BROLM_BF16 && out_dtype == BROLM_F32) return launch_norm<bf16, float>(a, n, s);
    if (w_dtype == BROLM_BF16 && out_dtype == BROLM_BF16) return launch_norm<bf16, bf16>(a, n, s);
    return BROLM_ERR_BAD_DTYPE;
}

}  // namespace

// x float rows of `hidden`; rows (int32 [n] or null) picks the input rows.
BROLM_API int brolm_layernorm(const void* x, const void* rows, const void* w, int w_dtype, float eps, void* out,
                              int out_dtype, int n, int hidden, cudaStream_t stream) {
    if (n <= 0) return BROLM_OK;
    if (hidden <= 0) return BROLM_ERR_BAD_SIZE;
    NormArgs a = {};
    a.x = (const float*)x; a.rows = (const int32_t*)rows; a.w = w; a.eps = eps; a.out = out; a.hidden = hidden;
    return launch_any(a, w_dtype, out_dtype, n, stream);
}

// h float [n][hidden], updated in place; w_post (null: y as it is) and w have one element type.
BROLM_API int brolm_residual_layernorm(void* h, const void* y, int n_parts, long long part_stride, const void* w_post,
                                       float eps_post, float off_post, const void* w, int w_dtype, float eps, void* out,
                                       int out_dtype, int n, int hidden, cudaStream_t stream) {
    if (n <= 0) return BROLM_OK;
    if (hidden <= 0 || n_parts < 1) return BROLM_ERR_BAD_SIZE;
    NormArgs a = {};
    a.h = (float*)h; a.y = (const float*)y; a.n_parts = n_parts; a.part_stride = part_stride;
    a.w_post = w_post; a.eps_post = eps_post; a.off_post = off_post; a.w = w; a.eps = eps; a.out = out; a.hidden = hidden;
    return launch_any(a, w_dtype, out_dtype, n, stream);
}
