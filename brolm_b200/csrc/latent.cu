// Latent attention, the row-wise step between the products and the attention kernel.  A token's projection row holds
// the compressed key/value row [a (R) | kr (dr)]; its queries, head by head [unrotated (dn) | rotated (dr)], lie in the
// same row or, when they come through a latent of their own, in rows of another product.  Each of three parts is made
// if its rows are given:
//
//   the latent row   [ a / sqrt(mean(a^2) + eps) * g  |  rot(kr, pos)  |  0 .. ]   (width Dp >= R + dr)
//   written to the packed rows of the step and to the token's place in the paged cache;
//   the rotated query parts  rot(qr_h, pos)  at columns R .. R + dr of head h of the
//   queries in latent space (width Dp per head; the first R columns come from the per-head
//   product with the keys' up-projection, the columns beyond R + dr are zero);
//   the queries' latent   cq = aq / sqrt(mean(aq^2) + eps) * gq   from Q columns of the projection row.
//
// With the queries in latent space the scores are plain dot products with the cached row,
// (q_n . W_uk c + q_r . k_r) = ((W_uk^T q_n) . c + q_r . k_r), and the cached row serves as the
// value as well (its first R columns, up-projected after the weighted sum).
//
// rot: the pairs of the first rd <= dr entries, (i, i + rd/2) or (2i, 2i + 1) ("interleaved"), turn by pos * f_i
// (cos and sin from a table built by the host); the entries beyond rd pass unchanged.
// The norms' statistics, the gains and the rotation are float; one rounding to the element type.
#include "common.cuh"

namespace {

template <typename T>
struct LatentArgs {
    const T* proj; long ld_proj;
    int kv_col;                          // where the compressed row starts (lat null: none)
    const T* q; long ld_q;               // query rows (qlat null: none)
    int cq_col, Q; const T* cq_gain; T* cq;       // the queries' latent (cq null: none), rows of Q
    const int32_t* positions; const float* cos_sin; int rd, inter;
    const T* gain; float eps; int heads, dn, dr, R, Dp;
    T* lat; T* qlat; T* pages; const int32_t* cache_rows;
};

template <typename T>
__global__ void __launch_bounds__(128) latent_rows_kernel(LatentArgs<T> p) {
    __shared__ float red[33];
    const int t = blockIdx.x;
    const int pos = p.positions[t];
    const T* row = p.proj + (size_t)t * p.ld_proj;
    const int half = p.rd >> 1;
    const float* cs = (pos >= 0 && p.cos_sin) ? p.cos_sin + (size_t)pos * half * 2 : nullptr;
    auto turned = [&](const T* v, int i) -> float {      // entry i of rot(v, pos)
        if (i >= p.rd || !cs) return to_float(v[i]);
        const int j = p.inter ? i >> 1 : (i < half ? i : i - half);
        const bool low = p.inter ? (i & 1) == 0 : i < half;
        const float c = cs[2 * j], s = cs[2 * j + 1];
        const float u = to_float(v[p.inter ? 2 * j : j]), w = to_float(v[p.inter ? 2 * j + 1 : j + half]);
        return low ? u * c - w * s : w * c + u * s;
    };
    if (p.cq) {
        const T* a = row + p.cq_col;
        float ss = 0.0f;
        for (int i = threadIdx.x; i < p.Q; i += blockDim.x) {
            const float v = to_float(a[i]);
            ss = fmaf(v, v, ss);
        }
        const float inv = rsqrtf(block_sum(ss, red) / (float)p.Q + p.eps);
        T* o = p.cq + (size_t)t * p.Q;
        for (int i = threadIdx.x; i < p.Q; i += blockDim.x) o[i] = from_float<T>(to_float(a[i]) * inv * to_float(p.cq_gain[i]));
    }
    if (p.lat) {
        const T* a = row + p.kv_col;
        float ss = 0.0f;
        for (int i = threadIdx.x; i < p.R; i += blockDim.x) {
            const float v = to_float(a[i]);
            ss = fmaf(v, v, ss);
        }
        ss = block_sum(ss, red);
        const float inv = rsqrtf(ss / (float)p.R + p.eps);
        const int cr = p.cache_rows ? p.cache_rows[t] : -1;
        T* l0 = p.lat + (size_t)t * p.Dp;
        T* l1 = (p.pages && cr >= 0 && pos >= 0) ? p.pages + (size_t)cr * p.Dp : nullptr;
        for (int i = threadIdx.x; i < p.Dp; i += blockDim.x) {
            float v = 0.0f;
            if (i < p.R) v = to_float(a[i]) * inv * to_float(p.gain[i]);
            else if (i < p.R + p.dr) v = turned(a + p.R, i - p.R);
            const T o = from_float<T>(v);
            l0[i] = o;
            if (l1) l1[i] = o;
        }
    }
    if (p.qlat) {
        const int tail = p.Dp - p.R;                     // columns R .. Dp of every head of the latent queries
        const T* q = p.q + (size_t)t * p.ld_q;
        for (int idx = threadIdx.x; idx < p.heads * tail; idx += blockDim.x) {
            const int h = idx / tail, i = idx - h * tail;
            const float v = i < p.dr ? turned(q + (size_t)h * (p.dn + p.dr) + p.dn, i) : 0.0f;
            p.qlat[((size_t)t * p.heads + h) * p.Dp + p.R + i] = from_float<T>(v);
        }
    }
}

template <typename T>
int launch_latent(const void* proj, long ld_proj, int kv_col, const void* q, long ld_q, int cq_col, int Q,
                  const void* cq_gain, void* cq, const void* positions, const void* cos_sin, int rd, int inter,
                  const void* gain, float eps, int heads, int dn, int dr, int R, int Dp, void* lat, void* qlat, void* pages,
                  const void* cache_rows, int tokens, cudaStream_t stream) {
    LatentArgs<T> p;
    p.proj = (const T*)proj; p.ld_proj = ld_proj; p.kv_col = kv_col; p.q = (const T*)q; p.ld_q = ld_q;
    p.cq_col = cq_col; p.Q = Q; p.cq_gain = (const T*)cq_gain; p.cq = (T*)cq;
    p.positions = (const int32_t*)positions; p.cos_sin = (const float*)cos_sin; p.rd = rd; p.inter = inter;
    p.gain = (const T*)gain; p.eps = eps; p.heads = heads; p.dn = dn; p.dr = dr; p.R = R; p.Dp = Dp;
    p.lat = (T*)lat; p.qlat = (T*)qlat; p.pages = (T*)pages; p.cache_rows = (const int32_t*)cache_rows;
    latent_rows_kernel<T><<<tokens, 128, 0, stream>>>(p);
    return launch_status();
}

}  // namespace

// lat, qlat, cq: each null when that part is not asked for.
BROLM_API int brolm_latent_rows(int dtype, const void* proj, long ld_proj, int kv_col, const void* q, long ld_q, int cq_col,
                                int Q, const void* cq_gain, void* cq, const void* positions, const void* cos_sin, int rd,
                                int inter, const void* gain, float eps, int heads, int dn, int dr, int R, int Dp, void* lat,
                                void* qlat, void* pages, const void* cache_rows, int tokens, cudaStream_t stream) {
    if (tokens <= 0) return BROLM_OK;
    if (heads <= 0 || dn < 0 || dr < 0 || R <= 0 || Dp < R + dr || rd < 0 || rd > dr || (rd & 1))
        return BROLM_ERR_BAD_SIZE;
    if ((cq && (Q <= 0 || !cq_gain)) || (lat && !gain) || (qlat && !q)) return BROLM_ERR_BAD_SIZE;
#define BROLM_LAT(T) launch_latent<T>(proj, ld_proj, kv_col, q, ld_q, cq_col, Q, cq_gain, cq, positions, cos_sin, rd, inter, \
                                      gain, eps, heads, dn, dr, R, Dp, lat, qlat, pages, cache_rows, tokens, stream)
    if (dtype == BROLM_F32) return BROLM_LAT(float);
    if (dtype == BROLM_BF16) return BROLM_LAT(bf16);
#undef BROLM_LAT
    return BROLM_ERR_BAD_DTYPE;
}
