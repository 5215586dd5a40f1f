// The gated delta rule as a recurrence over the packed tokens of a step (Yang et al., "Gated Delta Networks: Improving
// Mamba2 with Delta Rule").  Per head, with a state S of d x dv floats:
//
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
//
// H value heads of dv entries; G query/key heads of d entries, head h using q/k head h / (H / G).
//
// delta_rows makes the recurrence's inputs of a token from its projection row [q: G d | k: G d | v: H dv | zb: H | za: H]:
//     * a causal convolution over time per channel of q, k and v (K taps, column K - 1 the token's own; the K - 1
//       inputs before the step come from the rows the state keeps, zeros before the sequence's start), then silu;
//     * q and k as unit vectors per head, x / sqrt(sum(x^2) + norm_eps); q also times q_scale;
//     * beta = sigmoid(zb), and g - 1 = expm1(-exp(A_log) softplus(za + dt_bias)): a g close to one keeps in g - 1 the
//       digits that it loses itself when it is rounded to a float;
//     * q . k of every q/k head.
//   In a step of single tokens it also moves the kept inputs on (a prompt leaves that to conv_tail).
//
// delta_scan runs the recurrence.  With o = g S^T q + (q . k) u both sums over d are taken of the state as the token
// found it, so a token waits for one sum over a column (the one with k), and those with q are folded across the lanes
// sixteen tokens at once.  The state row of a sequence is laid out [head][value column][d padded to four], read at the
// start of the sequence's tokens of a step and written at their end; a row b with kv_len[b] <= 0 is padding.
//
// Everything is float arithmetic.
#include <type_traits>

#include "common.cuh"

namespace {

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

struct RowsArgs {
    const float* proj;        // [tokens][ldp]
    long ldp;
    const float* taps;        // [K][C] (tap-major), C = 2 G d + H dv
    int K, G, d, H, dv;
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
    int move_tail;            // every sequence brings one token: the kept inputs are moved on here
    float* u;                 // [tokens][ldu]: q | k | v
    long ldu;
    float* gates;             // [tokens][2 H]: (g - 1, beta) head by head
    float* qk;                // [tokens][G]
};

constexpr int ROWS_WARPS = 8;
constexpr int V_CHUNK = 128;  // value channels a warp takes at a time

// NJ: channels a lane holds of a q or k head (d <= 32 NJ).
template <int NJ>
__global__ void __launch_bounds__(ROWS_WARPS * 32) delta_rows_kernel(RowsArgs a) {
    pdl_trigger();
    const int t = blockIdx.x;
    const int pos = a.positions[t];
    if (pos < 0) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int b = a.tok_seq[t];
    const int q0 = a.cu_q[b], first = a.kv_len[b] - (a.cu_q[b + 1] - q0);
    const int K = a.K, qk_cols = a.G * a.d, v_cols = a.H * a.dv, C = 2 * qk_cols + v_cols;
    float* tail = a.state + (size_t)a.slots[b] * a.state_stride + a.tail_off;
    // tap j of channel c reads row_of(j)[c]
    auto row_of = [&](int j) -> const float* {
        const int q = pos - (K - 1) + j;
        return q >= first ? a.proj + (size_t)(q0 + q - first) * a.ldp : tail + (size_t)(q - first + K - 1) * C;
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
            for (int j = 0; j < K; ++j) {
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
            float sq = 0.0f, sk = 0.0f, dot = 0.0f;
#pragma unroll
            for (int n = 0; n < NJ; ++n) {
                q[n] = silu_f(q[n]);                    // silu(0) = 0: channels beyond d stay zero
                k[n] = silu_f(k[n]);
                sq = fmaf(q[n], q[n], sq);
                sk = fmaf(k[n], k[n], sk);
                dot = fmaf(q[n], k[n], dot);
            }
            sq = warp_sum(sq);
            sk = warp_sum(sk);
            dot = warp_sum(dot);
            const float iq = a.q_scale / sqrtf(sq + a.norm_eps), ik = 1.0f / sqrtf(sk + a.norm_eps);
#pragma unroll
            for (int n = 0; n < NJ; ++n) {
                const int c = lane + 32 * n;
                if (c < a.d) {
                    urow[cq + c] = q[n] * iq;
                    urow[ck + c] = k[n] * ik;
                }
            }
            if (lane == 0) a.qk[(size_t)t * a.G + unit] = dot * iq * ik;
            if (a.move_tail && K > 1) {
                for (int kk = 0; kk < K - 1; ++kk) {
                    const float* r = row_of(kk + 1);
                    float* dst = tail + (size_t)kk * C;
                    for (int c = lane; c < a.d; c += 32) {
                        const float x = r[cq + c], y = r[ck + c];
                        dst[cq + c] = x;
                        dst[ck + c] = y;
                    }
                }
            }
        } else if (unit < a.G + v_units) {
            const int c0 = 2 * qk_cols + (unit - a.G) * V_CHUNK;
            float v[V_CHUNK / 32];
#pragma unroll
            for (int n = 0; n < V_CHUNK / 32; ++n) v[n] = 0.0f;
            for (int j = 0; j < K; ++j) {
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
            if (a.move_tail && K > 1) {
                for (int kk = 0; kk < K - 1; ++kk) {
                    const float* r = row_of(kk + 1);
                    float* dst = tail + (size_t)kk * C;
                    for (int c = c0 + lane; c < min(c0 + V_CHUNK, C); c += 32) dst[c] = r[c];
                }
            }
        } else {
            const int h = (unit - a.G - v_units) * 32 + lane;
            if (h < a.H) {
                const float* z = a.proj + (size_t)t * a.ldp + C;
                const float dt = softplus_f(z[a.H + h] + a.dt_bias[h]);
                float2 g;
                g.x = expm1f(-expf(a.a_log[h]) * dt);
                g.y = 1.0f / (1.0f + expf(-z[h]));
                *reinterpret_cast<float2*>(a.gates + ((size_t)t * a.H + h) * 2) = g;
            }
        }
    }
}

struct ScanArgs {
    const float* u;           // [tokens][ld]: q | k | v
    long ld;
    const float* gates;       // [tokens][2 H]
    const float* qk;          // [tokens][G]
    int G, H, d, dv, dp;      // dp: d rounded up to a multiple of four
    const int32_t* cu_q;
    const int32_t* kv_len;
    const int32_t* slots;
    float* state;
    long state_stride;
    float* out;               // [tokens][ldo]; head h at h * dv
    long ldo;
    int ds;                   // lanes per value column (a power of two, at most 32)
    int vec;                  // every run of q, k and v starts at a multiple of 16 bytes
    int early;                // a step of single tokens: takes part in programmatic launch
};

constexpr int SCAN_TC = 16;

__device__ __forceinline__ void cp4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// A block of 128 threads takes one (sequence, head) and 128 / DS value columns; the DS lanes of a column keep NJ float4
// of the column's states each (entries 4 (j DS + ds) + e).  Tokens are staged sixteen at a time through two buffers.
// DSC > 0: lanes per column known to the compiler and NJ * DSC float4 are exactly a row of d; DSC = 0: any d.
template <int NJ, int DSC>
__global__ void __launch_bounds__(128) delta_scan_kernel(ScanArgs a) {
    extern __shared__ __align__(16) float sm[];
    if (a.early) pdl_trigger();
    constexpr bool EXACT = DSC > 0;
    const int DS = EXACT ? DSC : a.ds, VT = 128 / DS;
    const int dp = EXACT ? 4 * NJ * DSC : a.dp, dp4 = dp >> 2;
    const int stage = SCAN_TC * (2 * dp + VT + 4);    // q [TC][dp], k [TC][dp], v [TC][VT], (g - 1, beta, q.k, -) [TC]
    const int b = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * VT;
    const int kv_len = a.kv_len[b];
    if (kv_len <= 0) return;
    const int q0 = a.cu_q[b], q_len = a.cu_q[b + 1] - q0;
    if (q_len <= 0) return;
    const int hk = h / (a.H / a.G);
    const int ds = threadIdx.x % DS, vcol = threadIdx.x / DS, v = v0 + vcol;
    const bool live = v < a.dv;
    float* st = a.state + (size_t)a.slots[b] * a.state_stride + ((size_t)h * a.dv + (live ? v : 0)) * dp;
    float S[NJ * 4];
    // the state is this kernel's own: nothing that runs just before it in the step writes it
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        const int f = j * DS + ds;
        float4 s4 = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (live && f < dp4) s4 = *reinterpret_cast<const float4*>(st + 4 * f);
        S[4 * j] = s4.x; S[4 * j + 1] = s4.y; S[4 * j + 2] = s4.z; S[4 * j + 3] = s4.w;
    }
    // the padding of d to a multiple of four, and value columns beyond dv, stay zero in both buffers
    for (int i = threadIdx.x; i < 2 * stage; i += 128) sm[i] = 0.0f;
    __syncthreads();
    pdl_wait();
    const int n_chunks = (q_len + SCAN_TC - 1) / SCAN_TC;
    const int vt_here = min(VT, a.dv - v0);
    const int q_off = hk * a.d, k_off = a.G * a.d + hk * a.d, v_off = 2 * a.G * a.d + h * a.dv + v0;

    auto issue = [&](int chunk) {
        float* sq = sm + (chunk & 1) * stage;
        float* sk = sq + SCAN_TC * dp;
        float* sv = sk + SCAN_TC * dp;
        float* sg = sv + SCAN_TC * VT;
        const int t0 = chunk * SCAN_TC, n_tok = min(SCAN_TC, q_len - t0);
        if (a.vec) {
            const int d4 = a.d >> 2, v4 = vt_here >> 2;
            for (int idx = threadIdx.x; idx < n_tok * d4; idx += 128) {
                const int tt = idx / d4, c = (idx - tt * d4) << 2;
                const float* row = a.u + (size_t)(q0 + t0 + tt) * a.ld + c;
                cp16(sq + tt * dp + c, row + q_off);
                cp16(sk + tt * dp + c, row + k_off);
            }
            for (int idx = threadIdx.x; idx < n_tok * v4; idx += 128) {
                const int tt = idx / v4, c = (idx - tt * v4) << 2;
                cp16(sv + tt * VT + c, a.u + (size_t)(q0 + t0 + tt) * a.ld + v_off + c);
            }
        } else {
            for (int idx = threadIdx.x; idx < n_tok * a.d; idx += 128) {
                const int tt = idx / a.d, c = idx - tt * a.d;
                const float* row = a.u + (size_t)(q0 + t0 + tt) * a.ld + c;
                cp4(sq + tt * dp + c, row + q_off);
                cp4(sk + tt * dp + c, row + k_off);
            }
            for (int idx = threadIdx.x; idx < n_tok * vt_here; idx += 128) {
                const int tt = idx / vt_here, c = idx - tt * vt_here;
                cp4(sv + tt * VT + c, a.u + (size_t)(q0 + t0 + tt) * a.ld + v_off + c);
            }
        }
        for (int idx = threadIdx.x; idx < n_tok * 3; idx += 128) {
            const int tt = idx / 3, c = idx - tt * 3;
            const size_t t = (size_t)(q0 + t0 + tt);
            cp4(sg + tt * 4 + c, c < 2 ? a.gates + (t * a.H + h) * 2 + c : a.qk + t * a.G + hk);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    issue(0);
    for (int kc = 0; kc < n_chunks; ++kc) {
        const int t0 = kc * SCAN_TC, n_tok = min(SCAN_TC, q_len - t0);
        float* sq = sm + (kc & 1) * stage;
        float* sk = sq + SCAN_TC * dp;
        float* sv = sk + SCAN_TC * dp;
        const float4* sg = reinterpret_cast<const float4*>(sv + SCAN_TC * VT);
        if (kc + 1 < n_chunks) {
            issue(kc + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        float pv[SCAN_TC];                             // a lane's part of every token's result
        const float4* q4 = reinterpret_cast<const float4*>(sq) + ds;
        const float4* k4 = reinterpret_cast<const float4*>(sk) + ds;
        auto tokens = [&](auto full) {
#pragma unroll
            for (int tt = 0; tt < SCAN_TC; ++tt) {
                pv[tt] = 0.0f;
                if (decltype(full)::value || tt < n_tok) {
                    const float vv = sv[tt * VT + vcol];
                    const float4 g = sg[tt];
                    float4 kk[NJ];
                    float kx = 0.0f, ky = 0.0f, kz = 0.0f, kw = 0.0f, qx = 0.0f, qy = 0.0f, qz = 0.0f, qw = 0.0f;
#pragma unroll
                    for (int j = 0; j < NJ; ++j) {
                        if (EXACT || j * DS + ds < dp4) {
                            const float4 qq = q4[tt * dp4 + j * DS];
                            kk[j] = k4[tt * dp4 + j * DS];
                            kx = fmaf(S[4 * j], kk[j].x, kx);
                            ky = fmaf(S[4 * j + 1], kk[j].y, ky);
                            kz = fmaf(S[4 * j + 2], kk[j].z, kz);
                            kw = fmaf(S[4 * j + 3], kk[j].w, kw);
                            qx = fmaf(S[4 * j], qq.x, qx);
                            qy = fmaf(S[4 * j + 1], qq.y, qy);
                            qz = fmaf(S[4 * j + 2], qq.z, qz);
                            qw = fmaf(S[4 * j + 3], qq.w, qw);
                        } else {
                            kk[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                        }
                    }
                    float held = (kx + ky) + (kz + kw);                // what the column holds for k, summed over its lanes
#pragma unroll
                    for (int o = (EXACT ? DSC : 32) >> 1; o > 0; o >>= 1)
                        if (EXACT || o < DS) held += __shfl_xor_sync(0xffffffffu, held, o);
                    const float u = g.y * (vv - fmaf(g.x, held, held));
                    const float part = (qx + qy) + (qz + qw);
                    pv[tt] = fmaf(g.x, part, part) + (ds == 0 ? g.z * u : 0.0f);
#pragma unroll
                    for (int j = 0; j < NJ; ++j) {
                        S[4 * j] = fmaf(kk[j].x, u, fmaf(g.x, S[4 * j], S[4 * j]));
                        S[4 * j + 1] = fmaf(kk[j].y, u, fmaf(g.x, S[4 * j + 1], S[4 * j + 1]));
                        S[4 * j + 2] = fmaf(kk[j].z, u, fmaf(g.x, S[4 * j + 2], S[4 * j + 2]));
                        S[4 * j + 3] = fmaf(kk[j].w, u, fmaf(g.x, S[4 * j + 3], S[4 * j + 3]));
                    }
                }
            }
        };
        if (n_tok == SCAN_TC) tokens(std::true_type{});
        else tokens(std::false_type{});
        if (n_tok == 1) {                              // a single token: its sum alone crosses the lanes
            float acc = pv[0];
            for (int o = DS >> 1; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
            if (ds == 0 && live) a.out[(size_t)(q0 + t0) * a.ldo + (size_t)h * a.dv + v] = acc;
            __syncthreads();
            continue;
        }
        // The sixteen sums over a column's DS lanes, all at once: at every step a lane hands half of what it holds to
        // the lane `o` away and adds what it gets to the half it keeps.  `first` is the first token a lane ends up with.
        int first = 0, kept = SCAN_TC, o = DS >> 1;
#define BROLM_FOLD(N)                                                              \
        if (o > 0) {                                                               \
            const bool up = (ds & o) != 0;                                         \
            _Pragma("unroll") for (int i = 0; i < N; ++i) {                        \
                const float send = up ? pv[i] : pv[i + N];                         \
                const float keep = up ? pv[i + N] : pv[i];                         \
                pv[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);              \
            }                                                                      \
            if (up) first += N;                                                    \
            kept = N;                                                              \
            o >>= 1;                                                               \
        }
        BROLM_FOLD(8)
        BROLM_FOLD(4)
        BROLM_FOLD(2)
        BROLM_FOLD(1)
#undef BROLM_FOLD
        bool writer = live;
        if (o > 0) {                                   // 32 lanes a column: two lanes hold halves of one token's sum
            pv[0] += __shfl_xor_sync(0xffffffffu, pv[0], o);
            writer = writer && (ds & 1) == 0;
        }
        float* orow = a.out + (size_t)(q0 + t0 + first) * a.ldo + (size_t)h * a.dv + v;
#pragma unroll
        for (int i = 0; i < SCAN_TC; ++i)
            if (writer && i < kept && first + i < n_tok) orow[(size_t)i * a.ldo] = pv[i];
        __syncthreads();                               // the buffer is free for the chunk after the next
    }
    if (live) {
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const int f = j * DS + ds;
            if (f < dp4) *reinterpret_cast<float4*>(st + 4 * f) = make_float4(S[4 * j], S[4 * j + 1], S[4 * j + 2], S[4 * j + 3]);
        }
    }
}

template <int NJ, int DSC>
int launch_scan_as(const ScanArgs& a, dim3 grid, size_t smem, cudaStream_t stream) {
    static size_t allowed = 0;
    if (smem > 48 * 1024 && smem > allowed) {
        cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<NJ, DSC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        allowed = smem;
    }
    // a prompt's scan runs long on few warps: plain stream order, so that its blocks spread evenly over the SMs
    if (!a.early) return launch_in_order(delta_scan_kernel<NJ, DSC>, grid, dim3(128), smem, stream, a);
    return launch_pdl(delta_scan_kernel<NJ, DSC>, grid, dim3(128), smem, stream, a);
}

}  // namespace

// proj float [tokens][ldp]: q: G d | k: G d | v: H dv | zb: H | za: H; taps float [K][2 G d + H dv]; the state row holds
// the K - 1 kept inputs from tail_off on, [K - 1][2 G d + H dv].  u [tokens][ldu], gates [tokens][2 H], qk [tokens][G].
BROLM_API int brolm_delta_rows(const void* proj, long ldp, const void* taps, int K, int G, int d, int H, int dv,
                               float norm_eps, float q_scale, const void* a_log, const void* dt_bias, const void* tok_seq,
                               const void* positions, const void* cu_q, const void* kv_len, const void* slots, void* state,
                               long state_stride, long tail_off, int move_tail, void* u, long ldu, void* gates, void* qk,
                               int tokens, cudaStream_t stream) {
    if (tokens <= 0) return BROLM_OK;
    if (K < 1 || G <= 0 || d <= 0 || H <= 0 || H % G || dv <= 0) return BROLM_ERR_BAD_SIZE;
    if (d > 512) return BROLM_ERR_TOO_LARGE;
    if (((uintptr_t)gates & 7) != 0) return BROLM_ERR_ALIGNMENT;
    RowsArgs a;
    a.proj = (const float*)proj; a.ldp = ldp; a.taps = (const float*)taps; a.K = K; a.G = G; a.d = d; a.H = H; a.dv = dv;
    a.norm_eps = norm_eps; a.q_scale = q_scale; a.a_log = (const float*)a_log; a.dt_bias = (const float*)dt_bias;
    a.tok_seq = (const int32_t*)tok_seq; a.positions = (const int32_t*)positions; a.cu_q = (const int32_t*)cu_q;
    a.kv_len = (const int32_t*)kv_len; a.slots = (const int32_t*)slots; a.state = (float*)state;
    a.state_stride = state_stride; a.tail_off = tail_off; a.move_tail = move_tail;
    a.u = (float*)u; a.ldu = ldu; a.gates = (float*)gates; a.qk = (float*)qk;
    const int units = G + (H * dv + V_CHUNK - 1) / V_CHUNK + (H + 31) / 32;
    // few tokens: a unit a warp; many: a block walks a token's units
    int by = (units + ROWS_WARPS - 1) / ROWS_WARPS;
    if (by > 65535) by = 65535;
    dim3 grid(tokens, by);
    if (d <= 64) return launch_pdl(delta_rows_kernel<2>, grid, dim3(ROWS_WARPS * 32), 0, stream, a);
    if (d <= 128) return launch_pdl(delta_rows_kernel<4>, grid, dim3(ROWS_WARPS * 32), 0, stream, a);
    if (d <= 256) return launch_pdl(delta_rows_kernel<8>, grid, dim3(ROWS_WARPS * 32), 0, stream, a);
    return launch_pdl(delta_rows_kernel<16>, grid, dim3(ROWS_WARPS * 32), 0, stream, a);
}

// The state row of a sequence holds H * dv * round_up(d, 4) floats for this recurrence, from `state` on.
BROLM_API int brolm_delta_scan(const void* u, long ld, const void* gates, const void* qk, int G, int d, int H, int dv,
                               const void* cu_q, const void* kv_len, const void* slots, void* state, long state_stride,
                               void* out, long ldo, int batch, int max_q_len, cudaStream_t stream) {
    if (batch <= 0) return BROLM_OK;
    if (G <= 0 || d <= 0 || H <= 0 || H % G || dv <= 0) return BROLM_ERR_BAD_SIZE;
    if (H > 65535 || batch > 65535 || d > 512) return BROLM_ERR_TOO_LARGE;
    if (state_stride % 4 != 0 || ((uintptr_t)state & 15) != 0) return BROLM_ERR_ALIGNMENT;
    ScanArgs a;
    a.u = (const float*)u; a.ld = ld; a.gates = (const float*)gates; a.qk = (const float*)qk;
    a.G = G; a.H = H; a.d = d; a.dv = dv; a.dp = (d + 3) & ~3;
    a.cu_q = (const int32_t*)cu_q; a.kv_len = (const int32_t*)kv_len; a.slots = (const int32_t*)slots;
    a.state = (float*)state; a.state_stride = state_stride; a.out = (float*)out; a.ldo = ldo;
    a.vec = d % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && ((uintptr_t)u & 15) == 0;
    a.early = max_q_len == 1 ? 1 : 0;
    const int dp4 = a.dp >> 2, sms = device_sm_count();
    // a lane keeps nj float4 of a column's states, ds lanes a column; fewer states a lane (more, smaller blocks)
    // while the grid would leave SMs without a block
    auto lanes = [&](int nj) { int ds = 1; while (ds * nj < dp4) ds <<= 1; return ds; };
    auto blocks = [&](int nj) { const int vt = 128 / lanes(nj); return (long long)((dv + vt - 1) / vt) * H * batch; };
    int nj = 4;
    while (nj > 1 && lanes(nj) == 1 && nj / 2 >= dp4) nj >>= 1;
    while (nj > 1 && lanes(nj / 2) <= 32 && blocks(nj) < sms) nj >>= 1;
    const int ds = lanes(nj);
    if (ds > 32) return BROLM_ERR_TOO_LARGE;
    a.ds = ds;
    const int vt = 128 / ds;
    const size_t smem = (size_t)2 * SCAN_TC * (2 * a.dp + vt + 4) * sizeof(float);
    if (smem > 200 * 1024) return BROLM_ERR_TOO_LARGE;
    dim3 grid((dv + vt - 1) / vt, H, batch);
    // the sizes of real layers: everything about the row known to the compiler
    if (a.vec && nj * ds == dp4 && d == a.dp) {
        if (nj == 1 && ds == 8) return launch_scan_as<1, 8>(a, grid, smem, stream);
        if (nj == 2 && ds == 8) return launch_scan_as<2, 8>(a, grid, smem, stream);
        if (nj == 4 && ds == 4) return launch_scan_as<4, 4>(a, grid, smem, stream);
        if (nj == 4 && ds == 8) return launch_scan_as<4, 8>(a, grid, smem, stream);
        if (nj == 2 && ds == 16) return launch_scan_as<2, 16>(a, grid, smem, stream);
        if (nj == 4 && ds == 16) return launch_scan_as<4, 16>(a, grid, smem, stream);
    }
    if (nj == 1) return launch_scan_as<1, 0>(a, grid, smem, stream);
    if (nj == 2) return launch_scan_as<2, 0>(a, grid, smem, stream);
    return launch_scan_as<4, 0>(a, grid, smem, stream);
}
