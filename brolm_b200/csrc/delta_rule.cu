// The gated delta rule as a recurrence over the packed tokens of a step (Yang et al., "Gated Delta Networks: Improving
// Mamba2 with Delta Rule").  Per head, with a state S of d x dv floats:
//
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
//
// H value heads of dv entries; G query/key heads of d entries, head h using q/k head h / (H / G).  A token's projection
// row is [q: G d | k: G d | v: H dv | zb: H | za: H]; its inputs of the recurrence are
//     * q, k and v after a causal convolution over time per channel (K taps, the last one the token's own; zeros before
//       the sequence's start) and silu;
//     * q and k as unit vectors per head, x / sqrt(sum(x^2) + norm_eps); q also times q_scale;
//     * beta = sigmoid(zb), log g = -exp(A_log) softplus(za + dt_bias).
// The decay is kept as its logarithm and applied as S + expm1(log g) S: a g close to one keeps the digits that it loses
// itself when it is rounded to a float.
//
// A sequence's state row holds S as [head][value column][d padded to four] and, from tail_off on, the convolution's
// newest inputs as a ring of K rows, position p in row p mod K (no rows for K = 1): a step of single tokens reads K - 1
// rows and writes the one that no block of the launch reads.  A row b with kv_len[b] <= 0 is padding.
//
// A step of single tokens is one kernel, delta_step.  A prompt runs
//     delta_rows     the inputs of the recurrence, token by token;
//     delta_tail     the newest inputs into the ring;
//     delta_chunks   per sixteen tokens and head, what does not hang on the state;
//     delta_scan     the recurrence, sixteen tokens at a time.
// With S0 the state ahead of the sixteen tokens, D(i, j) the product of the decays of tokens j + 1 .. i and D(i) that of
// the tokens up to i, the recurrence's u solve a triangular system whose matrix needs the keys and gates alone:
//     u_i + sum_{j < i} beta_i D(i, j) (k_i . k_j) u_j = beta_i (v_i - D(i) S0^T k_i),       u = T (..)
//                                                      = U_i - S0^T w_i,   U = T (beta v),  w = T (beta D k)
//     o_i = D(i) S0^T q_i + sum_{j <= i} D(i, j) (q_i . k_j) u_j
//     S   = D(15) S0 + sum_j D(15, j) k_j u_j^T
// so all products with S0 of the sixteen tokens are independent of one another.  T's entries are at most one in
// magnitude (they are entries of products of contractions), every D is the exponential of a sum of its own.
//
// Everything is float arithmetic.
#include "common.cuh"

namespace {

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

typedef unsigned long long f32x2;          // two floats, for the paired multiply-add
__device__ __forceinline__ f32x2 pack2(float a, float b) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

struct DeltaArgs {
    const float* proj;        // [tokens][ldp]
    long ldp;
    const float* taps;        // [K][C] (tap-major), C = 2 G d + H dv
    int K, G, d, H, dv, dp;   // dp: d rounded up to a multiple of four
    float norm_eps, q_scale;
    const float* a_log;       // [H]
    const float* dt_bias;     // [H]
    const int32_t* tok_seq;
    const int32_t* positions;
    const int32_t* cu_q;
    const int32_t* kv_len;
    const int32_t* slots;
    float* state;
    long state_stride, tail_off;
    float* u;                 // [tokens][ldu]: q | k | v
    long ldu;
    float* gates;             // [tokens][2 H]: (log g, beta) head by head
    float* w;                 // [tokens][H dp]
    float* chunks;            // [chunk][H][REC]
    float* out;               // [tokens][ldo]; head h at h * dv
    long ldo;
    int tokens, vec;
};

__device__ __forceinline__ float log_decay(const DeltaArgs& a, float za, int h) {
    return -expf(a.a_log[h]) * softplus_f(za + a.dt_bias[h]);
}

// ---------------------------------------------------------------------------
// delta_rows, any sizes: a warp takes a unit (a q/k head, 128 value channels, or the gates of 32 heads) of a token.
// ---------------------------------------------------------------------------
constexpr int ROWS_WARPS = 8;
constexpr int V_CHUNK = 128;

template <int NJ>             // d <= 32 NJ
__global__ void __launch_bounds__(ROWS_WARPS * 32) delta_rows_kernel(DeltaArgs a) {
    pdl_trigger();
    const int t = blockIdx.x;
    const int pos = a.positions[t];
    if (pos < 0) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int b = a.tok_seq[t];
    const int q0 = a.cu_q[b], first = a.kv_len[b] - (a.cu_q[b + 1] - q0);
    const int K = a.K, qk_cols = a.G * a.d, v_cols = a.H * a.dv, C = 2 * qk_cols + v_cols;
    const float* ring = a.state + (size_t)a.slots[b] * a.state_stride + a.tail_off;
    const int j0 = max(0, K - 1 - pos);                    // taps ahead of it weigh positions before the start
    auto row_of = [&](int j) -> const float* {             // tap j of channel c reads row_of(j)[c]
        const int q = pos - (K - 1) + j;
        return q >= first ? a.proj + (size_t)(q0 + q - first) * a.ldp : ring + (size_t)(q % K) * C;
    };
    float* urow = a.u + (size_t)t * a.ldu;
    const int v_units = (v_cols + V_CHUNK - 1) / V_CHUNK, units = a.G + v_units + (a.H + 31) / 32;
    pdl_wait();
    for (int unit = blockIdx.y * ROWS_WARPS + warp; unit < units; unit += gridDim.y * ROWS_WARPS) {
        if (unit < a.G) {
            const int cq = unit * a.d, ck = qk_cols + unit * a.d;
            float q[NJ], k[NJ];
#pragma unroll
            for (int n = 0; n < NJ; ++n) q[n] = k[n] = 0.0f;
            for (int j = j0; j < K; ++j) {
                const float* r = row_of(j);
                const float* w = a.taps + (size_t)j * C;
#pragma unroll
                for (int n = 0; n < NJ; ++n) {
                    const int c = lane + 32 * n;
                    if (c < a.d) {
                        q[n] = fmaf(w[cq + c], r[cq + c], q[n]);
                        k[n] = fmaf(w[ck + c], r[ck + c], k[n]);
                    }
                }
            }
            float sq = 0.0f, sk = 0.0f;
#pragma unroll
            for (int n = 0; n < NJ; ++n) {
                q[n] = silu_f(q[n]);                        // silu(0) = 0: channels beyond d stay zero
                k[n] = silu_f(k[n]);
                sq = fmaf(q[n], q[n], sq);
                sk = fmaf(k[n], k[n], sk);
            }
            const float iq = a.q_scale / sqrtf(warp_sum(sq) + a.norm_eps), ik = 1.0f / sqrtf(warp_sum(sk) + a.norm_eps);
#pragma unroll
            for (int n = 0; n < NJ; ++n) {
                const int c = lane + 32 * n;
                if (c < a.d) {
                    urow[cq + c] = q[n] * iq;
                    urow[ck + c] = k[n] * ik;
                }
            }
        } else if (unit < a.G + v_units) {
            const int c0 = 2 * qk_cols + (unit - a.G) * V_CHUNK;
            float v[V_CHUNK / 32];
#pragma unroll
            for (int n = 0; n < V_CHUNK / 32; ++n) v[n] = 0.0f;
            for (int j = j0; j < K; ++j) {
                const float* r = row_of(j);
                const float* w = a.taps + (size_t)j * C;
#pragma unroll
                for (int n = 0; n < V_CHUNK / 32; ++n) {
                    const int c = c0 + lane + 32 * n;
                    if (c < C) v[n] = fmaf(w[c], r[c], v[n]);
                }
            }
#pragma unroll
            for (int n = 0; n < V_CHUNK / 32; ++n) {
                const int c = c0 + lane + 32 * n;
                if (c < C) urow[c] = silu_f(v[n]);
            }
        } else {
            const int h = (unit - a.G - v_units) * 32 + lane;
            if (h < a.H) {
                const float* z = a.proj + (size_t)t * a.ldp + C;
                float2 g;
                g.x = log_decay(a, z[a.H + h], h);
                g.y = 1.0f / (1.0f + expf(-z[h]));
                *reinterpret_cast<float2*>(a.gates + ((size_t)t * a.H + h) * 2) = g;
            }
        }
    }
}

// The same for up to four taps and sizes in fours: a warp takes its unit of a run of packed tokens, four channels a lane
// and load; where the run lies in one sequence all its rows are on their way before the first is used.
constexpr int RUN = 4, RUN_TAPS = 4;

__device__ __forceinline__ float4 fma4(float4 w, float4 x, float4 c) {
    return make_float4(fmaf(w.x, x.x, c.x), fmaf(w.y, x.y, c.y), fmaf(w.z, x.z, c.z), fmaf(w.w, x.w, c.w));
}
__device__ __forceinline__ float4 silu4(float4 v) { return make_float4(silu_f(v.x), silu_f(v.y), silu_f(v.z), silu_f(v.w)); }
__device__ __forceinline__ float dot4(float4 a, float4 b, float s) {
    return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, s))));
}
__device__ __forceinline__ float4 mul4(float4 a, float f) { return make_float4(a.x * f, a.y * f, a.z * f, a.w * f); }

// N columns of four channels a lane (col[n] < 0: none), the convolved and activated values handed to `use` per token.
template <int N, typename F>
__device__ __forceinline__ void run_of_tokens(const DeltaArgs& a, int C, const int (&col)[N], F use) {
    const int K = a.K, t0 = blockIdx.x * RUN, n_run = min(RUN, a.tokens - t0);
    const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    float4 w[RUN_TAPS][N];
#pragma unroll
    for (int jj = 0; jj < RUN_TAPS; ++jj)
#pragma unroll
        for (int n = 0; n < N; ++n) {
            const int j = jj - (RUN_TAPS - K);
            w[jj][n] = j >= 0 && col[n] >= 0 ? *reinterpret_cast<const float4*>(a.taps + (size_t)j * C + col[n]) : zero;
        }
    // rows m = 0 .. take tokens t - 3 + m of the sequence that token t (its position pos) belongs to
    auto fetch = [&](int t, int pos, int b, int m, float4 (&x)[N]) {
        const int first = a.kv_len[b] - (a.cu_q[b + 1] - a.cu_q[b]), q = pos - (RUN_TAPS - 1) + m;
        const bool in = q >= 0 && q > pos - K;
        const float* r = q >= first || !in ? a.proj + (size_t)(in ? t - (RUN_TAPS - 1) + m : t) * a.ldp
                                           : a.state + (size_t)a.slots[b] * a.state_stride + a.tail_off + (size_t)(q % K) * C;
#pragma unroll
        for (int n = 0; n < N; ++n) x[n] = in && col[n] >= 0 ? *reinterpret_cast<const float4*>(r + col[n]) : zero;
    };
    auto finish = [&](int t, const float4 (&x0)[N], const float4 (&x1)[N], const float4 (&x2)[N], const float4 (&x3)[N]) {
        float4 v[N];
#pragma unroll
        for (int n = 0; n < N; ++n)
            v[n] = silu4(fma4(w[3][n], x3[n], fma4(w[2][n], x2[n], fma4(w[1][n], x1[n], fma4(w[0][n], x0[n], zero)))));
        use(t, v);
    };
    const int b0 = a.tok_seq[t0], pos0 = a.positions[t0];
    const bool one = n_run == RUN && pos0 >= 0 && a.tok_seq[t0 + RUN - 1] == b0 && a.positions[t0 + RUN - 1] == pos0 + RUN - 1;
    pdl_wait();
    if (one) {
        float4 x[RUN + RUN_TAPS - 1][N];
#pragma unroll
        for (int m = 0; m < RUN_TAPS; ++m) fetch(t0, pos0, b0, m, x[m]);
#pragma unroll
        for (int m = RUN_TAPS; m < RUN + RUN_TAPS - 1; ++m)
#pragma unroll
            for (int n = 0; n < N; ++n)
                x[m][n] = col[n] >= 0 ? *reinterpret_cast<const float4*>(a.proj + (size_t)(t0 + m - (RUN_TAPS - 1)) * a.ldp + col[n]) : zero;
#pragma unroll
        for (int i = 0; i < RUN; ++i) finish(t0 + i, x[i], x[i + 1], x[i + 2], x[i + 3]);
        return;
    }
    for (int i = 0; i < n_run; ++i) {
        const int t = t0 + i, pos = a.positions[t];
        if (pos < 0) continue;
        const int b = a.tok_seq[t];
        float4 x[RUN_TAPS][N];
#pragma unroll
        for (int m = 0; m < RUN_TAPS; ++m) fetch(t, pos, b, m, x[m]);
        finish(t, x[0], x[1], x[2], x[3]);
    }
}

template <int NV>             // d <= 128 NV
__global__ void __launch_bounds__(ROWS_WARPS * 32) delta_rows_run_kernel(DeltaArgs a) {
    pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int qk_cols = a.G * a.d, v_cols = a.H * a.dv, C = 2 * qk_cols + v_cols;
    const int v_units = (v_cols + V_CHUNK - 1) / V_CHUNK, units = a.G + v_units + 1;
    const int unit = blockIdx.y * ROWS_WARPS + warp;
    if (unit >= units) return;
    if (unit < a.G) {
        int col[2 * NV];
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int c = lane * 4 + 128 * n;
            col[n] = c < a.d ? unit * a.d + c : -1;
            col[NV + n] = c < a.d ? qk_cols + unit * a.d + c : -1;
        }
        run_of_tokens<2 * NV>(a, C, col, [&](int t, const float4 (&v)[2 * NV]) {
            float sq = 0.0f, sk = 0.0f;
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                sq = dot4(v[n], v[n], sq);
                sk = dot4(v[NV + n], v[NV + n], sk);
            }
            const float iq = a.q_scale / sqrtf(warp_sum(sq) + a.norm_eps), ik = 1.0f / sqrtf(warp_sum(sk) + a.norm_eps);
            float* urow = a.u + (size_t)t * a.ldu;
#pragma unroll
            for (int n = 0; n < NV; ++n)
                if (col[n] >= 0) {
                    *reinterpret_cast<float4*>(urow + col[n]) = mul4(v[n], iq);
                    *reinterpret_cast<float4*>(urow + col[NV + n]) = mul4(v[NV + n], ik);
                }
        });
    } else if (unit < a.G + v_units) {
        const int c = 2 * qk_cols + (unit - a.G) * V_CHUNK + lane * 4;
        const int col[1] = {c < C ? c : -1};
        run_of_tokens<1>(a, C, col, [&](int t, const float4 (&v)[1]) {
            if (col[0] >= 0) *reinterpret_cast<float4*>(a.u + (size_t)t * a.ldu + col[0]) = v[0];
        });
    } else {
        pdl_wait();
        const int t0 = blockIdx.x * RUN, n = min(RUN, a.tokens - t0) * a.H;
        for (int i = lane; i < n; i += 32) {
            const int t = t0 + i / a.H, h = i % a.H;
            if (a.positions[t] < 0) continue;
            const float* z = a.proj + (size_t)t * a.ldp + C;
            float2 g;
            g.x = log_decay(a, z[a.H + h], h);
            g.y = 1.0f / (1.0f + expf(-z[h]));
            *reinterpret_cast<float2*>(a.gates + ((size_t)t * a.H + h) * 2) = g;
        }
    }
}

// ring[p mod K][c] <- the input of position p, for the newest K - 1 positions of every sequence (after all that read it).
__global__ void __launch_bounds__(256) delta_tail_kernel(DeltaArgs a) {
    pdl_trigger();
    const int b = blockIdx.x, C = 2 * a.G * a.d + a.H * a.dv;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    const int kv_len = a.kv_len[b];
    if (kv_len <= 0 || c >= C) return;
    const int q0 = a.cu_q[b], first = kv_len - (a.cu_q[b + 1] - q0);
    float* ring = a.state + (size_t)a.slots[b] * a.state_stride + a.tail_off;
    pdl_wait();
    for (int p = max(first, kv_len - (a.K - 1)); p < kv_len; ++p)
        ring[(size_t)(p % a.K) * C + c] = a.proj[(size_t)(q0 + p - first) * a.ldp + c];
}

// ---------------------------------------------------------------------------
// A step of single tokens: convolution, unit norms, gates and the recurrence.  A block of 128 threads takes one
// (sequence, head) and 128 / DS value columns; the DS lanes of a column keep NJ float4 of its states each (entries
// 4 (j DS + ds) + e).  Every block of a head makes the head's q and k (a channel or a few per thread).
// ---------------------------------------------------------------------------
template <int NJ, int DS>
__global__ void __launch_bounds__(128) delta_step_kernel(DeltaArgs a) {
    constexpr int DP = 4 * NJ * DS, VT = 128 / DS, CH = (DP + 127) / 128;
    __shared__ __align__(16) float sq[DP], sk[DP];
    __shared__ float sv[VT], red[3][4];
    pdl_trigger();
    const int b = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * VT;
    const int kv_len = a.kv_len[b];
    if (kv_len <= 0) return;
    const int t = a.cu_q[b], pos = kv_len - 1, K = a.K;
    const int share = a.H / a.G, hk = h / share;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int ds = tid % DS, vcol = tid / DS, v = v0 + vcol;
    const bool live = v < a.dv;
    const int dp4 = a.dp >> 2, qk_cols = a.G * a.d, C = 2 * qk_cols + a.H * a.dv;
    float* row = a.state + (size_t)a.slots[b] * a.state_stride;
    float* st = row + ((size_t)h * a.dv + (live ? v : 0)) * a.dp;
    float* ring = row + a.tail_off;
    // The state and the kept inputs were written by the step before: they are fetched, and the convolution's older taps
    // summed, while the product ahead of this kernel finishes.
    float4 S[NJ];
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        const int f = j * DS + ds;
        S[j] = live && f < dp4 ? *reinterpret_cast<const float4*>(st + 4 * f) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    float aq[CH], ak[CH], av = 0.0f;
#pragma unroll
    for (int n = 0; n < CH; ++n) aq[n] = ak[n] = 0.0f;
    const int cq = hk * a.d, ck = qk_cols + hk * a.d, cv = 2 * qk_cols + h * a.dv + v0 + tid;
    const bool own_v = tid < VT && v0 + tid < a.dv;
    for (int j = max(0, K - 1 - pos); j < K - 1; ++j) {
        const float* r = ring + (size_t)((pos - (K - 1) + j) % K) * C;
        const float* w = a.taps + (size_t)j * C;
#pragma unroll
        for (int n = 0; n < CH; ++n) {
            const int c = tid + 128 * n;
            if (c < a.d) {
                aq[n] = fmaf(w[cq + c], r[cq + c], aq[n]);
                ak[n] = fmaf(w[ck + c], r[ck + c], ak[n]);
            }
        }
        if (own_v) av = fmaf(w[cv], r[cv], av);
    }
    const float* w = a.taps + (size_t)(K - 1) * C;
    float wq[CH], wk[CH];
#pragma unroll
    for (int n = 0; n < CH; ++n) {
        const int c = tid + 128 * n;
        wq[n] = c < a.d ? w[cq + c] : 0.0f;
        wk[n] = c < a.d ? w[ck + c] : 0.0f;
    }
    const float wv = own_v ? w[cv] : 0.0f, neg_a = -expf(a.a_log[h]), dtb = a.dt_bias[h];
    pdl_wait();
    const float* x = a.proj + (size_t)t * a.ldp;
    float* keep = ring + (size_t)(pos % K) * C;
    const bool keeps_qk = K > 1 && blockIdx.x == 0 && h == hk * share;
    const float zb = x[C + h], za = x[C + a.H + h];
    float s0 = 0.0f, s1 = 0.0f, s2 = 0.0f;
#pragma unroll
    for (int n = 0; n < CH; ++n) {
        const int c = tid + 128 * n;
        if (c < a.d) {
            const float xq = x[cq + c], xk = x[ck + c];
            const float q = silu_f(fmaf(wq[n], xq, aq[n])), k = silu_f(fmaf(wk[n], xk, ak[n]));
            sq[c] = q;
            sk[c] = k;
            s0 = fmaf(q, q, s0);
            s1 = fmaf(k, k, s1);
            s2 = fmaf(q, k, s2);
            if (keeps_qk) { keep[cq + c] = xq; keep[ck + c] = xk; }
        } else if (c < DP) {
            sq[c] = sk[c] = 0.0f;
        }
    }
    if (own_v) {
        const float xv = x[cv];
        sv[tid] = silu_f(fmaf(wv, xv, av));
        if (K > 1) keep[cv] = xv;
    }
    s0 = warp_sum(s0);
    s1 = warp_sum(s1);
    s2 = warp_sum(s2);
    if (lane == 0) { red[0][warp] = s0; red[1][warp] = s1; red[2][warp] = s2; }
    const float gm1 = expm1f(neg_a * softplus_f(za + dtb)), beta = 1.0f / (1.0f + expf(-zb));
    __syncthreads();
    const float iq = a.q_scale / sqrtf((red[0][0] + red[0][1]) + (red[0][2] + red[0][3]) + a.norm_eps);
    const float ik = 1.0f / sqrtf((red[1][0] + red[1][1]) + (red[1][2] + red[1][3]) + a.norm_eps);
    const float qk = ((red[2][0] + red[2][1]) + (red[2][2] + red[2][3])) * iq * ik;
    float held = 0.0f, read = 0.0f;                        // S^T k and S^T q of the column, before the decay
    float4 kk[NJ];
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        kk[j] = reinterpret_cast<const float4*>(sk)[j * DS + ds];
        const float4 qq = reinterpret_cast<const float4*>(sq)[j * DS + ds];
        held = dot4(S[j], kk[j], held);
        read = dot4(S[j], qq, read);
    }
#pragma unroll
    for (int o = DS >> 1; o > 0; o >>= 1) {
        held += __shfl_xor_sync(0xffffffffu, held, o);
        read += __shfl_xor_sync(0xffffffffu, read, o);
    }
    held *= ik;
    read *= iq;
    const float u = beta * ((live ? sv[vcol] : 0.0f) - fmaf(gm1, held, held)), ku = ik * u;
    if (live) {
        if (ds == 0) a.out[(size_t)t * a.ldo + (size_t)h * a.dv + v] = fmaf(qk, u, fmaf(gm1, read, read));
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const int f = j * DS + ds;
            if (f < dp4) {
                S[j].x = fmaf(kk[j].x, ku, fmaf(gm1, S[j].x, S[j].x));
                S[j].y = fmaf(kk[j].y, ku, fmaf(gm1, S[j].y, S[j].y));
                S[j].z = fmaf(kk[j].z, ku, fmaf(gm1, S[j].z, S[j].z));
                S[j].w = fmaf(kk[j].w, ku, fmaf(gm1, S[j].w, S[j].w));
                *reinterpret_cast<float4*>(st + 4 * f) = S[j];
            }
        }
    }
}

// ---------------------------------------------------------------------------
// delta_chunks: a block takes sixteen tokens of one (sequence, head).  It writes w (rows of dp, zeros beyond d), puts U in
// v's place and leaves a record of REC floats:
//   B [16][20] (rows padded against bank conflicts), B_ij = D(i, j) (q_i . k_j) for j <= i,
//   D(i) [16], D(15, i) [16], expm1(log D(15)), three unused.
// Tokens beyond the sequence's end have k = q = v = 0, log g = 0 and beta = 0, and change nothing.
// Record number of chunk c of sequence b: cu_q[b] / 16 + b + c (sequences never share one).
// ---------------------------------------------------------------------------
constexpr int TC = 16, MR = 20, OFF_V = TC * MR, REC = OFF_V + 2 * TC + 4;

__device__ __forceinline__ int record_of(int q0, int b, int chunk) { return q0 / TC + b + chunk; }

__global__ void __launch_bounds__(128) delta_chunks_kernel(DeltaArgs a) {
    extern __shared__ __align__(16) float sm[];            // k [16][ld], q [16][ld]
    __shared__ float lg[TC], be[TC], A[TC][TC + 1];
    __shared__ __align__(16) float Tb[TC][MR], Tk[TC][MR]; // T beta and T beta D
    const int chunk = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
    const int q0 = a.cu_q[b], q_len = a.cu_q[b + 1] - q0, t0 = chunk * TC;
    if (a.kv_len[b] <= 0 || t0 >= q_len) return;
    const int n_tok = min(TC, q_len - t0), hk = h / (a.H / a.G), ld = a.dp + 4, dp4 = a.dp >> 2;
    float* sk = sm;
    float* sq = sm + TC * ld;
    float* rec = a.chunks + ((size_t)record_of(q0, b, chunk) * a.H + h) * REC;
    if (a.vec) {
        for (int i = tid; i < TC * dp4; i += 128) {
            const int r = i / dp4, c = (i - r * dp4) * 4;
            float4 k = make_float4(0.0f, 0.0f, 0.0f, 0.0f), q = k;
            if (r < n_tok) {
                const float* row = a.u + (size_t)(q0 + t0 + r) * a.ldu + hk * a.d + c;
                q = *reinterpret_cast<const float4*>(row);
                k = *reinterpret_cast<const float4*>(row + a.G * a.d);
            }
            *reinterpret_cast<float4*>(sk + r * ld + c) = k;
            *reinterpret_cast<float4*>(sq + r * ld + c) = q;
        }
    } else {
        for (int i = tid; i < TC * a.dp; i += 128) {
            const int r = i / a.dp, c = i - r * a.dp;
            const bool in = r < n_tok && c < a.d;
            const float* row = a.u + (size_t)(q0 + t0 + (in ? r : 0)) * a.ldu + hk * a.d + (in ? c : 0);
            sk[r * ld + c] = in ? row[a.G * a.d] : 0.0f;
            sq[r * ld + c] = in ? row[0] : 0.0f;
        }
    }
    if (tid < TC) {
        const float2 g = tid < n_tok ? *reinterpret_cast<const float2*>(a.gates + ((size_t)(q0 + t0 + tid) * a.H + h) * 2)
                                     : make_float2(0.0f, 0.0f);
        lg[tid] = g.x;
        be[tid] = g.y;
    }
    __syncthreads();
    // thread (i, jj): the products of row i with rows jj and jj + 8
    const int i = tid >> 3, jj = tid & 7;
    float kk[2] = {0.0f, 0.0f}, qk[2] = {0.0f, 0.0f};
    for (int f = 0; f < dp4; ++f) {
        const float4 ki = *reinterpret_cast<const float4*>(sk + i * ld + 4 * f), qi = *reinterpret_cast<const float4*>(sq + i * ld + 4 * f);
#pragma unroll
        for (int m = 0; m < 2; ++m) {
            const float4 kj = *reinterpret_cast<const float4*>(sk + (jj + 8 * m) * ld + 4 * f);
            kk[m] = dot4(ki, kj, kk[m]);
            qk[m] = dot4(qi, kj, qk[m]);
        }
    }
#pragma unroll
    for (int m = 0; m < 2; ++m) {
        const int j = jj + 8 * m;
        float s = 0.0f;
        for (int l = j + 1; l <= i; ++l) s += lg[l];
        const float D = i >= j ? expf(s) : 0.0f;
        A[i][j] = i > j ? be[i] * D * kk[m] : 0.0f;
        rec[i * MR + j] = D * qk[m];
        if (i == TC - 1) rec[OFF_V + TC + j] = D;
        if (j == 0) {
            rec[OFF_V + i] = expf(s + lg[0]);
            if (i == TC - 1) rec[OFF_V + 2 * TC] = expm1f(s + lg[0]);
        }
    }
    __syncthreads();
    if (tid < TC) {                                        // column tid of T, from the diagonal down
        float x[TC], s_all = 0.0f;
        for (int l = 0; l <= tid; ++l) s_all += lg[l];
        const float fb = be[tid], fk = fb * expf(s_all);
#pragma unroll
        for (int r = 0; r < TC; ++r) {
            float s = 0.0f;
#pragma unroll
            for (int j = 0; j < r; ++j) s = fmaf(A[r][j], x[j], s);
            x[r] = r < tid ? 0.0f : r == tid ? 1.0f : -s;
        }
#pragma unroll
        for (int r = 0; r < TC; ++r) {
            Tb[r][tid] = x[r] * fb;
            Tk[r][tid] = x[r] * fk;
        }
    }
    __syncthreads();
    // a column of k, or of v, a thread: sixteen sums over the sixteen tokens
    for (int c = tid; c < a.dp + a.dv; c += 128) {
        const bool is_k = c < a.dp;
        const int cv = c - a.dp;
        float* vcol = a.u + (size_t)(q0 + t0) * a.ldu + 2 * a.G * a.d + h * a.dv + cv;
        float x[TC];
#pragma unroll
        for (int j = 0; j < TC; ++j) x[j] = is_k ? sk[j * ld + c] : (j < n_tok ? vcol[(size_t)j * a.ldu] : 0.0f);
        float* dst = is_k ? a.w + (size_t)(q0 + t0) * a.H * a.dp + h * a.dp + c : vcol;
        const size_t step = is_k ? (size_t)a.H * a.dp : (size_t)a.ldu;
        const float* m = is_k ? &Tk[0][0] : &Tb[0][0];
#pragma unroll
        for (int r = 0; r < TC; ++r) {
            float y = 0.0f;
#pragma unroll
            for (int j = 0; j <= r; ++j) y = fmaf(m[r * MR + j], x[j], y);
            if (r < n_tok) dst[(size_t)r * step] = y;
        }
    }
}

// ---------------------------------------------------------------------------
// delta_scan: a block of 256 threads takes one (sequence, head) and sixteen value columns, sixteen tokens at a time.  A
// warp holds an eighth of d for all sixteen columns, a lane NJ x 4 entries of d (f = (warp NJ + j) 4 + lane mod 4 counts
// fours of d) for two columns.  With two warps a scheduler one issues while the other waits.
//   1. partial products of w and q with the state, folded across the four lanes of a column pair, left per warp;
//   2. the eight warps' parts joined: u = U - S0^T w (warps 0 to 3), D S0^T q (warps 4 to 7);
//   3. the state's update by all, o by warps 4 to 7.
// The rows come through three stages of cp.async.
// ---------------------------------------------------------------------------
__device__ __forceinline__ void cp4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

constexpr int VC = 16;                                     // value columns of a block
constexpr int PR = 20;                                     // floats between two rows of sixteen columns
// w, q, k rows [16][DP], U [16][PR], the record
template <int NJ> __host__ __device__ constexpr int scan_stage() { return 3 * TC * 128 * NJ + TC * PR + REC; }
template <int NJ> __host__ __device__ constexpr int scan_stages() { return NJ == 4 ? 2 : 3; }
constexpr int SCAN_WARPS = 8, SCAN_THREADS = 32 * SCAN_WARPS;
template <int NJ> __host__ __device__ constexpr int scan_floats() {
    return scan_stages<NJ>() * scan_stage<NJ>() + SCAN_WARPS * 2 * TC * PR + 2 * TC * PR;
}

// EXACT: d is DP, every row is copied in fours and all sixteen columns are there: the copies' indices are shifts.
template <int NJ, bool EXACT>
__global__ void __launch_bounds__(SCAN_THREADS) delta_scan_kernel(DeltaArgs a) {
    extern __shared__ __align__(16) float sm[];
    constexpr int DP = 128 * NJ, STAGE = scan_stage<NJ>(), STAGES = scan_stages<NJ>();
    const int b = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * VC;
    const int kv_len = a.kv_len[b];
    if (kv_len <= 0) return;
    const int q0 = a.cu_q[b], q_len = a.cu_q[b + 1] - q0;
    if (q_len <= 0) return;
    const int hk = h / (a.H / a.G), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int ds = lane & 3, cg = lane >> 2;               // place in d, pair of columns
    const int dp4 = EXACT ? DP / 4 : a.dp >> 2, vt = EXACT ? VC : min(VC, a.dv - v0);
    float* part = sm + STAGES * STAGE;                     // [8 warps][32 rows][PR]
    float* us = part + SCAN_WARPS * 2 * TC * PR;                 // [16][PR] u
    float* ud = us + TC * PR;                              // [16][PR] D(15, j) u_j
    f32x2 S[NJ][2][2];
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        const int f = (warp * NJ + j) * 4 + ds;
#pragma unroll
        for (int c = 0; c < 2; ++c) {
            const int v = 2 * cg + c;
            float4 s4 = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (v < vt && f < dp4)
                s4 = *reinterpret_cast<const float4*>(a.state + (size_t)a.slots[b] * a.state_stride + ((size_t)h * a.dv + v0 + v) * a.dp + 4 * f);
            S[j][c][0] = pack2(s4.x, s4.y);
            S[j][c][1] = pack2(s4.z, s4.w);
        }
    }
    const int n_chunks = (q_len + TC - 1) / TC;
    // rows padded to DP, value columns beyond dv and tokens beyond the end read as zeros
    if (!EXACT || (q_len & (TC - 1))) {
        for (int i = tid; i < STAGES * STAGE; i += SCAN_THREADS) sm[i] = 0.0f;
        __syncthreads();
    }
    const int q_off = hk * a.d, k_off = a.G * a.d + hk * a.d, v_off = 2 * a.G * a.d + h * a.dv + v0;
    auto issue = [&](int chunk) {
        float* sw = sm + (chunk % STAGES) * STAGE;
        float* sq = sw + TC * DP;
        float* sk = sq + TC * DP;
        float* sv = sk + TC * DP;
        const int t0 = chunk * TC, n_tok = min(TC, q_len - t0);
        if (n_tok < TC && chunk >= STAGES) {               // the last stage holds older tokens where there are none now
            for (int i = tid; i < (TC - n_tok) * DP; i += SCAN_THREADS)
                sw[n_tok * DP + i] = sq[n_tok * DP + i] = sk[n_tok * DP + i] = 0.0f;
            for (int i = tid; i < (TC - n_tok) * PR; i += SCAN_THREADS) sv[n_tok * PR + i] = 0.0f;
        }
        for (int idx = tid; idx < n_tok * dp4; idx += SCAN_THREADS) {
            const int tt = idx / dp4, c = (idx - tt * dp4) << 2;
            cp16(sw + tt * DP + c, a.w + (size_t)(q0 + t0 + tt) * a.H * a.dp + h * a.dp + c);
        }
        if (EXACT || a.vec) {
            const int d4 = EXACT ? DP / 4 : a.d >> 2, v4 = vt >> 2;
            for (int idx = tid; idx < n_tok * d4; idx += SCAN_THREADS) {
                const int tt = idx / d4, c = (idx - tt * d4) << 2;
                const float* row = a.u + (size_t)(q0 + t0 + tt) * a.ldu + c;
                cp16(sq + tt * DP + c, row + q_off);
                cp16(sk + tt * DP + c, row + k_off);
            }
            for (int idx = tid; idx < n_tok * v4; idx += SCAN_THREADS) {
                const int tt = idx / v4, c = (idx - tt * v4) << 2;
                cp16(sv + tt * PR + c, a.u + (size_t)(q0 + t0 + tt) * a.ldu + v_off + c);
            }
        } else {
            for (int idx = tid; idx < n_tok * a.d; idx += SCAN_THREADS) {
                const int tt = idx / a.d, c = idx - tt * a.d;
                const float* row = a.u + (size_t)(q0 + t0 + tt) * a.ldu + c;
                cp4(sq + tt * DP + c, row + q_off);
                cp4(sk + tt * DP + c, row + k_off);
            }
            for (int idx = tid; idx < n_tok * vt; idx += SCAN_THREADS) {
                const int tt = idx / vt, c = idx - tt * vt;
                cp4(sv + tt * PR + c, a.u + (size_t)(q0 + t0 + tt) * a.ldu + v_off + c);
            }
        }
        const float* rec = a.chunks + ((size_t)record_of(q0, b, chunk) * a.H + h) * REC;
        for (int idx = tid; idx < REC / 4; idx += SCAN_THREADS) cp16(sv + TC * PR + 4 * idx, rec + 4 * idx);
    };
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s) {
        if (s < n_chunks) issue(s);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    const int jrow = tid >> 3, jcg = tid & 7;              // phase 2: row (of 32) and pair of columns
    const bool out2 = vt == VC && a.dv % 2 == 0 && a.ldo % 2 == 0 && ((uintptr_t)a.out & 7) == 0;
    for (int kc = 0; kc < n_chunks; ++kc) {
        asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
        __syncthreads();                                   // this stage has landed, and no warp works on the one before
        if (kc + STAGES - 1 < n_chunks) issue(kc + STAGES - 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        const float* sw = sm + (kc % STAGES) * STAGE;      // w rows, q rows behind them
        const float* sk = sw + 2 * TC * DP;
        const float* sv = sk + TC * DP;
        const float* sr = sv + TC * PR;
#pragma unroll
        for (int g = 0; g < 4; ++g) {                      // eight rows at a time; lane ds ends up with rows 2 ds, 2 ds + 1
            float s[8][2];
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                f32x2 acc[2][2] = {{0ull, 0ull}, {0ull, 0ull}};
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const ulonglong2 x = reinterpret_cast<const ulonglong2*>(sw + (8 * g + r) * DP)[(warp * NJ + j) * 4 + ds];
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        acc[c][0] = fma2(S[j][c][0], x.x, acc[c][0]);
                        acc[c][1] = fma2(S[j][c][1], x.y, acc[c][1]);
                    }
                }
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    const float2 e = unpack2(acc[c][0]), f = unpack2(acc[c][1]);
                    s[r][c] = (e.x + e.y) + (f.x + f.y);
                }
            }
            // at every step a lane hands half of the rows it holds to the lane `o` away and adds what it gets to the rest
#pragma unroll
            for (int n = 4, o = 2; o > 0; n >>= 1, o >>= 1) {
                const bool up = (ds & o) != 0;
#pragma unroll
                for (int r = 0; r < 4; ++r)
                    if (r < n) {
#pragma unroll
                        for (int c = 0; c < 2; ++c) {
                            const float send = up ? s[r][c] : s[r + n][c], keep = up ? s[r + n][c] : s[r][c];
                            s[r][c] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                        }
                    }
            }
#pragma unroll
            for (int r = 0; r < 2; ++r)
                *reinterpret_cast<float2*>(part + (warp * 2 * TC + 8 * g + 2 * ds + r) * PR + 2 * cg) = make_float2(s[r][0], s[r][1]);
        }
        __syncthreads();
        float2 y = make_float2(0.0f, 0.0f);
#pragma unroll
        for (int w = 0; w < SCAN_WARPS; ++w) {
            const float2 x = *reinterpret_cast<const float2*>(part + (w * 2 * TC + jrow) * PR + 2 * jcg);
            y.x += x.x; y.y += x.y;
        }
        const int tok = jrow & (TC - 1);
        if (jrow < TC) {
            const float2 U = *reinterpret_cast<const float2*>(sv + tok * PR + 2 * jcg);
            const float f = sr[OFF_V + TC + tok];
            y = make_float2(U.x - y.x, U.y - y.y);
            *reinterpret_cast<float2*>(us + tok * PR + 2 * jcg) = y;
            *reinterpret_cast<float2*>(ud + tok * PR + 2 * jcg) = make_float2(y.x * f, y.y * f);
        }
        __syncthreads();
        const float dm1 = sr[OFF_V + 2 * TC];
        float st[NJ][2][4];
#pragma unroll
        for (int j = 0; j < NJ; ++j)
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                const float2 e = unpack2(S[j][c][0]), f = unpack2(S[j][c][1]);
                st[j][c][0] = fmaf(dm1, e.x, e.x);
                st[j][c][1] = fmaf(dm1, e.y, e.y);
                st[j][c][2] = fmaf(dm1, f.x, f.x);
                st[j][c][3] = fmaf(dm1, f.y, f.y);
            }
#pragma unroll
        for (int t = 0; t < TC; ++t) {
            const float2 u2 = *reinterpret_cast<const float2*>(ud + t * PR + 2 * cg);
            const float uu[2] = {u2.x, u2.y};
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
                const float4 k = *reinterpret_cast<const float4*>(sk + t * DP + 4 * ((warp * NJ + j) * 4 + ds));
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    st[j][c][0] = fmaf(k.x, uu[c], st[j][c][0]);
                    st[j][c][1] = fmaf(k.y, uu[c], st[j][c][1]);
                    st[j][c][2] = fmaf(k.z, uu[c], st[j][c][2]);
                    st[j][c][3] = fmaf(k.w, uu[c], st[j][c][3]);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < NJ; ++j)
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                S[j][c][0] = pack2(st[j][c][0], st[j][c][1]);
                S[j][c][1] = pack2(st[j][c][2], st[j][c][3]);
            }
        const int t = kc * TC + tok;
        if (jrow >= TC && t < q_len) {
            const float f = sr[OFF_V + tok];
            y.x *= f; y.y *= f;
#pragma unroll
            for (int j = 0; j < TC; j += 4) {
                const float4 m = *reinterpret_cast<const float4*>(sr + tok * MR + j);
                const float mm[4] = {m.x, m.y, m.z, m.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float2 u2 = *reinterpret_cast<const float2*>(us + (j + e) * PR + 2 * jcg);
                    y.x = fmaf(mm[e], u2.x, y.x);
                    y.y = fmaf(mm[e], u2.y, y.y);
                }
            }
            float* o = a.out + (size_t)(q0 + t) * a.ldo + (size_t)h * a.dv + v0 + 2 * jcg;
            if (out2) {
                *reinterpret_cast<float2*>(o) = y;
            } else {
                if (2 * jcg < vt) o[0] = y.x;
                if (2 * jcg + 1 < vt) o[1] = y.y;
            }
        }
    }
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        const int f = (warp * NJ + j) * 4 + ds;
#pragma unroll
        for (int c = 0; c < 2; ++c) {
            const int v = 2 * cg + c;
            const float2 e = unpack2(S[j][c][0]), g = unpack2(S[j][c][1]);
            if (v < vt && f < dp4)
                *reinterpret_cast<float4*>(a.state + (size_t)a.slots[b] * a.state_stride + ((size_t)h * a.dv + v0 + v) * a.dp + 4 * f) =
                    make_float4(e.x, e.y, g.x, g.y);
        }
    }
}

template <int NJ, bool EXACT>
int launch_scan_as(const DeltaArgs& a, int batch, cudaStream_t stream) {
    constexpr size_t smem = scan_floats<NJ>() * sizeof(float);
    static_assert(smem <= 227 * 1024, "the stages do not fit an SM");
    static bool raised = false;
    if (!raised) {
        cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<NJ, EXACT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        raised = true;
    }
    // plain stream order: it runs long on few warps, which are to spread evenly over the SMs
    return launch_in_order(delta_scan_kernel<NJ, EXACT>, dim3((a.dv + VC - 1) / VC, a.H, batch), dim3(SCAN_THREADS), smem, stream, a);
}

template <int NJ>
int launch_scan(const DeltaArgs& a, int batch, cudaStream_t stream) {
    return a.vec && a.d == 128 * NJ && a.dv % VC == 0 ? launch_scan_as<NJ, true>(a, batch, stream)
                                                      : launch_scan_as<NJ, false>(a, batch, stream);
}

template <int NJ, int DS>
int launch_step(const DeltaArgs& a, int batch, cudaStream_t stream) {
    const int vt = 128 / DS;
    return launch_pdl(delta_step_kernel<NJ, DS>, dim3((a.dv + vt - 1) / vt, a.H, batch), dim3(128), 0, stream, a);
}

int check_sizes(const DeltaArgs& a, int batch) {
    if (a.K < 1 || a.G <= 0 || a.d <= 0 || a.H <= 0 || a.H % a.G || a.dv <= 0) return BROLM_ERR_BAD_SIZE;
    if (a.H > 65535 || batch > 65535 || a.d > 512) return BROLM_ERR_TOO_LARGE;
    if (a.state_stride % 4 != 0 || ((uintptr_t)a.state & 15) != 0) return BROLM_ERR_ALIGNMENT;
    return BROLM_OK;
}

// lanes of a column and float4 a lane for a row of d
int step_by_size(const DeltaArgs& a, int batch, cudaStream_t stream) {
    if (a.dp <= 32) return launch_step<1, 8>(a, batch, stream);
    if (a.dp <= 64) return launch_step<2, 8>(a, batch, stream);
    if (a.dp <= 128) return launch_step<4, 8>(a, batch, stream);
    if (a.dp <= 256) return launch_step<4, 16>(a, batch, stream);
    return launch_step<8, 16>(a, batch, stream);
}
int scan_by_size(const DeltaArgs& a, int batch, cudaStream_t stream) {
    if (a.dp <= 128) return launch_scan<1>(a, batch, stream);
    if (a.dp <= 256) return launch_scan<2>(a, batch, stream);
    return launch_scan<4>(a, batch, stream);
}

}  // namespace

// Floats of one chunk's record of one head.
BROLM_API int brolm_delta_record() { return REC; }

// One token per sequence.  proj float [tokens][ldp], taps float [K][2 G d + H dv]; the state row of a sequence holds
// H * dv * round_up(d, 4) floats from `state` on and the ring of kept inputs from tail_off on.  out [tokens][ldo].
BROLM_API int brolm_delta_step(const void* proj, long ldp, const void* taps, int K, int G, int d, int H, int dv, float norm_eps,
                               float q_scale, const void* a_log, const void* dt_bias, const void* cu_q, const void* kv_len,
                               const void* slots, void* state, long state_stride, long tail_off, void* out, long ldo,
                               int batch, cudaStream_t stream) {
    if (batch <= 0) return BROLM_OK;
    DeltaArgs a = {};
    a.proj = (const float*)proj; a.ldp = ldp; a.taps = (const float*)taps;
    a.K = K; a.G = G; a.d = d; a.H = H; a.dv = dv; a.dp = (d + 3) & ~3;
    a.norm_eps = norm_eps; a.q_scale = q_scale; a.a_log = (const float*)a_log; a.dt_bias = (const float*)dt_bias;
    a.cu_q = (const int32_t*)cu_q; a.kv_len = (const int32_t*)kv_len; a.slots = (const int32_t*)slots;
    a.state = (float*)state; a.state_stride = state_stride; a.tail_off = tail_off; a.out = (float*)out; a.ldo = ldo;
    const int bad = check_sizes(a, batch);
    return bad ? bad : step_by_size(a, batch, stream);
}

// Any number of tokens per sequence, four kernels (three for K = 1).  u [tokens][ldu] (ldu a multiple of four), gates
// [tokens][2 H], w [tokens][H * round_up(d, 4)] and chunks [tokens / 16 + batch + 1][H][REC] are scratch, 16-byte aligned.
BROLM_API int brolm_delta_prompt(const void* proj, long ldp, const void* taps, int K, int G, int d, int H, int dv,
                                 float norm_eps, float q_scale, const void* a_log, const void* dt_bias, const void* tok_seq,
                                 const void* positions, const void* cu_q, const void* kv_len, const void* slots, void* state,
                                 long state_stride, long tail_off, void* u, long ldu, void* gates, void* w, void* chunks, void* out,
                                 long ldo, int tokens, int batch, int max_q_len, cudaStream_t stream) {
    if (batch <= 0 || tokens <= 0) return BROLM_OK;
    DeltaArgs a = {};
    a.proj = (const float*)proj; a.ldp = ldp; a.taps = (const float*)taps;
    a.K = K; a.G = G; a.d = d; a.H = H; a.dv = dv; a.dp = (d + 3) & ~3;
    a.norm_eps = norm_eps; a.q_scale = q_scale; a.a_log = (const float*)a_log; a.dt_bias = (const float*)dt_bias;
    a.tok_seq = (const int32_t*)tok_seq; a.positions = (const int32_t*)positions;
    a.cu_q = (const int32_t*)cu_q; a.kv_len = (const int32_t*)kv_len; a.slots = (const int32_t*)slots;
    a.state = (float*)state; a.state_stride = state_stride; a.tail_off = tail_off;
    a.u = (float*)u; a.ldu = ldu; a.gates = (float*)gates; a.w = (float*)w; a.chunks = (float*)chunks; a.out = (float*)out; a.ldo = ldo;
    a.tokens = tokens;
    const int bad = check_sizes(a, batch);
    if (bad) return bad;
    if (max_q_len <= 0) return BROLM_ERR_BAD_SIZE;
    if (ldu % 4 != 0 || (((uintptr_t)u | (uintptr_t)gates | (uintptr_t)w | (uintptr_t)chunks) & 15)) return BROLM_ERR_ALIGNMENT;
    const int C = 2 * G * d + H * dv, v_units = (H * dv + V_CHUNK - 1) / V_CHUNK;
    a.vec = d % 4 == 0 && dv % 4 == 0;
    int st;
    if (a.vec && K <= RUN_TAPS && d <= 256 && ldp % 4 == 0 && tail_off % 4 == 0 &&
        (((uintptr_t)proj | (uintptr_t)taps) & 15) == 0) {
        dim3 grid((tokens + RUN - 1) / RUN, (G + v_units + 1 + ROWS_WARPS - 1) / ROWS_WARPS);
        st = d <= 128 ? launch_pdl(delta_rows_run_kernel<1>, grid, dim3(ROWS_WARPS * 32), 0, stream, a)
                      : launch_pdl(delta_rows_run_kernel<2>, grid, dim3(ROWS_WARPS * 32), 0, stream, a);
    } else {
        int by = (G + v_units + (H + 31) / 32 + ROWS_WARPS - 1) / ROWS_WARPS;
        if (by > 65535) by = 65535;
        dim3 grid(tokens, by);
        st = d <= 64    ? launch_pdl(delta_rows_kernel<2>, grid, dim3(ROWS_WARPS * 32), 0, stream, a)
             : d <= 128 ? launch_pdl(delta_rows_kernel<4>, grid, dim3(ROWS_WARPS * 32), 0, stream, a)
             : d <= 256 ? launch_pdl(delta_rows_kernel<8>, grid, dim3(ROWS_WARPS * 32), 0, stream, a)
                        : launch_pdl(delta_rows_kernel<16>, grid, dim3(ROWS_WARPS * 32), 0, stream, a);
    }
    if (st) return st;
    if (K > 1) {
        st = launch_pdl(delta_tail_kernel, dim3(batch, (C + 255) / 256), dim3(256), 0, stream, a);
        if (st) return st;
    }
    const size_t smem = (size_t)2 * TC * (a.dp + 4) * sizeof(float);
    if (smem > 48 * 1024) {
        static bool raised = false;
        if (!raised) {
            const int most = 2 * TC * (512 + 4) * (int)sizeof(float);
            cudaError_t e = cudaFuncSetAttribute(delta_chunks_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
            if (e != cudaSuccess) return (int)e;
            raised = true;
        }
    }
    st = launch_in_order(delta_chunks_kernel, dim3((max_q_len + TC - 1) / TC, H, batch), dim3(128), smem, stream, a);
    if (st) return st;
    return scan_by_size(a, batch, stream);
}
