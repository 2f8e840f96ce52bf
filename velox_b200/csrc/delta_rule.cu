// The gated delta rule: per head a state S [D, Dv] that forgets, and that a token corrects instead of adding to:
//   S' = g_t S_(t-1);  u_t = beta_t (v_t - S'^T k_t);  S_t = S' + k_t u_t^T;  o_t = S_t^T q_t
// with q, k, v behind a short causal convolution over time (per channel, then silu), q and k unit vectors per head, a decay
// g = exp(-exp(A_log) softplus(a + dt_bias)) and a step size beta = sigmoid(b) per head and token.  Several heads may share
// one q/k head.
//
//   delta_conv      convolution, silu and unit vectors of a step's tokens (float32 out)
//   delta_coef      decays, step sizes, and what follows from them and from the products among keys and queries within
//                   eight tokens
//   delta_walk      the recurrence over a step's tokens; afterwards the last inputs of the convolutions go into their slots
//   delta_decode    a step of single tokens: all of this, the norm of every head's output and its gate in one kernel
//
// State per request (float32): S transposed, [H, Dv, D] (a column of S is contiguous), and the last inputs of the
// convolutions as a ring [taps, channels]: position p lies in row p mod taps.  A token at position p reads rows p - 1 ..
// p - taps + 1 and writes row p, which is none of those, so the blocks of a decode step need no order among them.  Rows of
// positions before 0 count as zeros and are never read.  Channels are numbered q [G, D], k [G, D], v [H, Dv].
#include "tcgen05_gemm.cuh"

#define DR_EPS_UNIT 1e-6f
#define DR_MINI 8      // tokens of a mini-chunk
#define DR_COEF 20     // numbers per token and head that the walk reads
#define DR_MAX_TAPS 64

__device__ __forceinline__ float dr_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float dr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// VEC consecutive elements of a row as floats.
template <int VEC> __device__ __forceinline__ void dr_load(const float* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    } else if constexpr (VEC == 2) {
        const float2 a = *reinterpret_cast<const float2*>(p);
        v[0] = a.x; v[1] = a.y;
    } else {
        v[0] = *p;
    }
}
template <int VEC> __device__ __forceinline__ void dr_load(const bf16* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
    } else if constexpr (VEC == 2) {
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
        v[0] = a.x; v[1] = a.y;
    } else {
        v[0] = __bfloat162float(*p);
    }
}
template <int VEC> __device__ __forceinline__ void dr_store(float* p, const float (&v)[VEC]) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else if constexpr (VEC == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
    else *p = v[0];
}

// What the convolution of one token needs to know about where it stands.
struct DrPlace {
    int local;        // its row among the rows that its request brings
    int pos;          // its position
    const float* ring;
};
__device__ __forceinline__ DrPlace dr_place(int t, const int* seq_of_token, const int* cu_seqlens, const int* state_slots,
                                            const int* positions, const float* ring, size_t ring_size) {
    const int seq = seq_of_token[t];
    return DrPlace{t - cu_seqlens[seq], positions[t], ring + (size_t)state_slots[seq] * ring_size};
}

// ---- convolution, silu, unit vectors ----
// What the walk reads, in runs that one bulk copy brings: qk float32 [G, tokens, 2, DP] (q as a unit vector times q_mul, k as a
// unit vector, zeros from D up to DP: 64, 128 or 256) and v float32 [H, ceil(Dv / 8), tokens, 8] (what lies past Dv is left alone).
__host__ __device__ constexpr int dr_padded(int D) { return D <= 64 ? 64 : (D <= 128 ? 128 : 256); }
// Where channel c of token t goes (c counts q [G, D], k [G, D], v [H, Dv]).
__device__ __forceinline__ float* dr_target(float* qk, float* v, int t, int c, int tokens, int G, int D, int DP, int Dv) {
    if (c < 2 * G * D) {
        const int is_k = c >= G * D, r = c - is_k * G * D, g = r / D;
        return qk + (((size_t)g * tokens + t) * 2 + is_k) * DP + (r - g * D);
    }
    const int r = c - 2 * G * D, h = r / Dv, col = r - h * Dv;
    return v + (((size_t)h * ((Dv + 7) >> 3) + (col >> 3)) * tokens + t) * 8 + (col & 7);
}

// The convolution of VEC channels from c on of token t, each tap's row from the step or from the ring.
template <typename T, int VEC>
__device__ __forceinline__ void dr_conv_at(const T* __restrict__ x, int ldx, const float* __restrict__ w, int C, int taps, int t,
                                           const DrPlace& at, int c, float (&out)[VEC]) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) out[e] = 0.f;
    for (int j = min(taps - 1, at.pos); j >= 0; --j) {
        float v[VEC], wv[VEC];
        if (at.local >= j) dr_load<VEC>(x + (size_t)(t - j) * ldx + c, v);
        else dr_load<VEC>(at.ring + (size_t)((at.pos - j) % taps) * C + c, v);
        dr_load<VEC>(w + (size_t)(taps - 1 - j) * C + c, wv);
#pragma unroll
        for (int e = 0; e < VEC; ++e) out[e] = fmaf(wv[e], v[e], out[e]);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) out[e] = dr_silu(out[e]);
}

// Any sizes (D up to 256): a warp takes one unit (a q or k head, or a run of v's channels) of one token.
template <typename T>
__global__ void __launch_bounds__(128)
delta_conv_any_kernel(const T* __restrict__ x, int ldx, const float* __restrict__ w, const float* __restrict__ ring,
                      const int* __restrict__ seq_of_token, const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots,
                      const int* __restrict__ positions, float* __restrict__ qk, float* __restrict__ vout, int tokens, int G, int D, int H, int Dv,
                      int taps, float q_mul, int units) {
    pdl_wait();
    pdl_trigger();
    const long long id = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    const int t = (int)(id / units), unit = (int)(id - (long long)t * units);
    if (t >= tokens) return;
    const int C = 2 * G * D + H * Dv, DP = dr_padded(D);
    const DrPlace at = dr_place(t, seq_of_token, cu_seqlens, state_slots, positions, ring, (size_t)taps * C);
    const bool is_v = unit >= 2 * G;
    const int c0 = is_v ? 2 * G * D + (unit - 2 * G) * 256 : unit * D, n = is_v ? min(256, C - c0) : D;
    float v[8], ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        float one[1] = {0.f};
        if (lane + 32 * i < n) dr_conv_at<T, 1>(x, ldx, w, C, taps, t, at, c0 + lane + 32 * i, one);
        v[i] = one[0];
        ss = fmaf(v[i], v[i], ss);
    }
    const float mul = is_v ? 1.f : rsqrtf(warp_sum(ss) + DR_EPS_UNIT) * (unit < G ? q_mul : 1.f);
#pragma unroll
    for (int i = 0; i < 8; ++i)
        if (lane + 32 * i < n) *dr_target(qk, vout, t, c0 + lane + 32 * i, tokens, G, D, DP, Dv) = v[i] * mul;
    if (!is_v) {
        float* row = dr_target(qk, vout, t, c0, tokens, G, D, DP, Dv);
        for (int d = D + lane; d < DP; d += 32) row[d] = 0.f;
    }
}

// The same for four taps and heads of 32 VEC channels, a warp taking DR_RUN consecutive tokens of a unit.  Where all of them
// and the three before the first belong to one request and to this step, every row is asked for before the first is used and
// read once, not once a tap; else token by token.
#define DR_RUN 8
template <typename T, int VEC>
__global__ void __launch_bounds__(128)
delta_conv_run_kernel(const T* __restrict__ x, int ldx, const float* __restrict__ w, const float* __restrict__ ring,
                      const int* __restrict__ seq_of_token, const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots,
                      const int* __restrict__ positions, float* __restrict__ qk, float* __restrict__ vout, int tokens, int G, int H, int Dv,
                      float q_mul, int units) {
    constexpr int TAPS = 4, D = 32 * VEC, DP = dr_padded(D);
    const int C = 2 * G * D + H * Dv;
    const int lane = threadIdx.x & 31;
    const long long id = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    const int unit = (int)(id % units), t0 = (int)(id / units) * DR_RUN;
    if (t0 >= tokens) return;   // (a warp past the end; a block's first warp never is)
    const int c = unit * D + lane * VEC;   // (v's channels follow those of the 2 G heads of q and k)
    const bool live = c < C, is_v = unit >= 2 * G;
    const float unit_mul = unit < G ? q_mul : 1.f;
    float wt[TAPS][VEC];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) wt[j][e] = 0.f;
        if (live) dr_load<VEC>(w + (size_t)j * C + c, wt[j]);
    }
    pdl_wait();
    pdl_trigger();
    const int seq = seq_of_token[t0], first = cu_seqlens[seq], last = cu_seqlens[seq + 1];
    float* const target = live ? dr_target(qk, vout, t0, c, tokens, G, D, DP, Dv) - (size_t)t0 * (is_v ? 8 : 2 * DP) : nullptr;
    auto finish = [&](int t, float (&o)[VEC]) {
        if (!is_v) {   // (a warp holds one unit)
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < VEC; ++e) ss = fmaf(o[e], o[e], ss);
            const float mul = rsqrtf(warp_sum(ss) + DR_EPS_UNIT) * unit_mul;
#pragma unroll
            for (int e = 0; e < VEC; ++e) o[e] *= mul;
        }
        if (live) dr_store<VEC>(target + (size_t)t * (is_v ? 8 : 2 * DP), o);
        if (D < DP && !is_v) target[(size_t)t * 2 * DP + D] = 0.f;   // (heads of 32: a lane's channel, and the pad beside it)
    };
    if (t0 - first >= TAPS - 1 && t0 + DR_RUN <= last) {
        float win[DR_RUN + TAPS - 1][VEC];
#pragma unroll
        for (int i = 0; i < DR_RUN + TAPS - 1; ++i) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) win[i][e] = 0.f;
            if (live) dr_load<VEC>(x + (size_t)(t0 - (TAPS - 1) + i) * ldx + c, win[i]);
        }
#pragma unroll
        for (int u = 0; u < DR_RUN; ++u) {
            float o[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                float s = wt[0][e] * win[u][e];
#pragma unroll
                for (int j = 1; j < TAPS; ++j) s = fmaf(wt[j][e], win[u + j][e], s);
                o[e] = dr_silu(s);
            }
            finish(t0 + u, o);
        }
        return;
    }
    for (int t = t0; t < min(t0 + DR_RUN, tokens); ++t) {
        const DrPlace at = dr_place(t, seq_of_token, cu_seqlens, state_slots, positions, ring, (size_t)TAPS * C);
        float o[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) o[e] = 0.f;
        if (live) dr_conv_at<T, VEC>(x, ldx, w, C, TAPS, t, at, c, o);
        finish(t, o);
    }
}

template <typename T>
static int launch_delta_conv(const T* x, int ldx, const float* w, const float* ring, const int* seq_of_token, const int* cu_seqlens,
                             const int* state_slots, const int* positions, float* qk, float* v, int tokens, int G, int D, int H, int Dv, int taps,
                             float q_mul, cudaStream_t stream) {
    const int HDv = H * Dv, vec = D / 32, C = 2 * G * D + HDv;
    const bool run = taps == 4 && (D == 32 || D == 64 || D == 128) && tokens > 1 && Dv % vec == 0 && ldx % vec == 0 &&
                     !(((uintptr_t)x | (uintptr_t)w | (uintptr_t)ring) & 15) && C % vec == 0;
    const int units = 2 * G + (run ? (HDv + D - 1) / D : (HDv + 255) / 256);
    const long long warps = (long long)units * (run ? (tokens + DR_RUN - 1) / DR_RUN : tokens);
    if ((warps + 3) / 4 > 0x7fffffffLL) return VX_ERR_LIMIT;
    const unsigned blocks = (unsigned)((warps + 3) / 4);
#define DR_GO(V_) VX_LAUNCH_K(VX_K_ELEMENTWISE, (delta_conv_run_kernel<T, V_>), blocks, 128, 0, stream, x, ldx, w, ring, seq_of_token, \
                              cu_seqlens, state_slots, positions, qk, v, tokens, G, H, Dv, q_mul, units)
    if (run && vec == 1) DR_GO(1);
    else if (run && vec == 2) DR_GO(2);
    else if (run) DR_GO(4);
    else
        VX_LAUNCH_K(VX_K_ELEMENTWISE, (delta_conv_any_kernel<T>), blocks, 128, 0, stream, x, ldx, w, ring, seq_of_token, cu_seqlens,
                    state_slots, positions, qk, v, tokens, G, D, H, Dv, taps, q_mul, units);
#undef DR_GO
    VX_LAUNCH_CHECK();
    return VX_OK;
}

// x [tokens, ldx]: the projections q [G, D], k [G, D], v [H, Dv] from column 0 on.  w float32 [taps, C] (the last row is the
// current token's), ring float32 [slots, taps, C] (read only).  qk, v: see above, 16-byte aligned.
extern "C" int vx_delta_conv(const void* x, int ldx, const float* w, const float* ring, const int* seq_of_token,
                             const int* cu_seqlens, const int* state_slots, const int* positions, float* qk, float* v, int tokens,
                             int G, int D, int H, int Dv, int taps, float q_mul, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return VX_OK;
    if (G <= 0 || D <= 0 || H <= 0 || Dv <= 0 || H % G || taps <= 0 || ldx < 2 * G * D + H * Dv) return VX_ERR_SHAPE;
    if (D > 256 || taps > DR_MAX_TAPS) return VX_ERR_LIMIT;
    if (((uintptr_t)qk | (uintptr_t)v) & 15) return VX_ERR_ALIGN;
    if (dtype == VX_F32)
        return launch_delta_conv<float>((const float*)x, ldx, w, ring, seq_of_token, cu_seqlens, state_slots, positions, qk, v, tokens, G,
                                        D, H, Dv, taps, q_mul, stream);
    if (dtype == VX_BF16)
        return launch_delta_conv<bf16>((const bf16*)x, ldx, w, ring, seq_of_token, cu_seqlens, state_slots, positions, qk, v, tokens, G, D,
                                       H, Dv, taps, q_mul, stream);
    return VX_ERR_DTYPE;
}

// ---- the coefficients of a mini-chunk ----
// A request's rows of this step are taken DR_MINI at a time.  With gamma_i the product of the decays g up to token i of the
// mini-chunk, rho_ij that of the decays after j up to i, A_ij = beta_i rho_ij (k_i . k_j) for j < i and S the state before the
// mini-chunk, the rule unrolls to
//   (I + A) u = r,  r_i = beta_i v_i - beta_i gamma_i (k_i . S)
//   o_i = gamma_i (q_i . S) + sum_(j <= i) rho_ij (q_i . k_j) u_j
//   S  <- gamma_last S + sum_j rho_(last,j) k_j u_j^T
// Per token i and head: beta_i, beta_i gamma_i, gamma_i, rho_(last,i), then row i of (I + A)^-1, then the rho_ij (q_i . k_j).
// A warp per eight token rows and q/k head; the products are summed over the lanes all 64 together (two rounds of 32).
// Tokens past a request's last count as k = q = 0, beta = 0, g = 1.

// 8 CC sums over 32 lanes (CC 1, 2 or 4): in the first rounds half of the values change sides, then what lanes are left is added;
// lane l ends with the sum number l mod 8 CC.  The order of a sum's additions does not depend on CC.  With PERMUTED lane l
// brings the value 8 c + (s xor (l mod 8)) in p[8 c + s]: then what changes sides in the first three rounds is in the same
// place for every lane, and nothing has to be selected.
template <int CC, bool PERMUTED>
__device__ __forceinline__ float dr_sums(float (&p)[8 * CC], int lane) {
#pragma unroll
    for (int n = 4; n > 0; n >>= 1) {
        const bool hi = lane & n;
#pragma unroll
        for (int c = 0; c < CC; ++c)
#pragma unroll
            for (int i = 0; i < n; ++i) {
                const float keep = !PERMUTED && hi ? p[8 * c + n + i] : p[8 * c + i], give = !PERMUTED && hi ? p[8 * c + i] : p[8 * c + n + i];
                p[8 * c + i] = keep + __shfl_xor_sync(0xffffffffu, give, n);
            }
    }
#pragma unroll
    for (int n = 1; n < 4; n <<= 1) {   // lanes 8 n apart, columns n apart
        const bool hi = lane & (8 * n);
        if (n < CC) {
#pragma unroll
            for (int c = 0; c < CC; c += 2 * n) {
                const float keep = hi ? p[8 * (c + (n < CC ? n : 0))] : p[8 * c], give = hi ? p[8 * c] : p[8 * (c + (n < CC ? n : 0))];
                p[8 * c] = keep + __shfl_xor_sync(0xffffffffu, give, 8 * n);
            }
        } else {
            p[0] += __shfl_xor_sync(0xffffffffu, p[0], 8 * n);
        }
    }
    return p[0];
}

#define DR_CW 4   // warps of a block
__global__ void __launch_bounds__(DR_CW * 32)
delta_coef_kernel(const float* __restrict__ qkv, const float* __restrict__ ab, int ldab, int a_col, int b_col,
                  const float* __restrict__ neg_exp_a, const float* __restrict__ dt_bias, const int* __restrict__ seq_of_token,
                  const int* __restrict__ cu_seqlens, float* __restrict__ coef, int tokens, int G, int D, int H) {
    __shared__ float kk_s[DR_CW][64], qk_s[DR_CW][64], a_s[DR_CW][4][64];
    pdl_wait();
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, i = lane & 7;
    const long long id = (long long)blockIdx.x * DR_CW + warp;
    const int kvh = (int)(id % G);
    const long long row0 = id / G * DR_MINI;
    float *kk = kk_s[warp], *qk = qk_s[warp];
    // (among eight rows of the step a mini-chunk starts once, or more often where requests end)
    for (int u = 0; u < DR_MINI; ++u) {
        if (row0 + u >= tokens) break;
        const int t = (int)row0 + u, seq = seq_of_token[t];
        if ((t - cu_seqlens[seq]) % DR_MINI != 0) continue;
        const int n = min(DR_MINI, cu_seqlens[seq + 1] - t);
        // products: 28 of keys (j < i) in one round of 32, 36 of queries and keys (j <= i) in the rest
        float pk[32], pq[32], px[4];
#pragma unroll
        for (int v = 0; v < 32; ++v) { pk[v] = 0.f; pq[v] = 0.f; }
#pragma unroll
        for (int v = 0; v < 4; ++v) px[v] = 0.f;
        for (int d = lane; d < D; d += 32) {
            float kr[DR_MINI], qr[DR_MINI];
#pragma unroll
            for (int r = 0; r < DR_MINI; ++r) {
                const float* src = qkv + ((size_t)kvh * tokens + t + r) * 2 * dr_padded(D) + d;
                qr[r] = r < n ? src[0] : 0.f;
                kr[r] = r < n ? src[dr_padded(D)] : 0.f;
            }
#pragma unroll
            for (int a = 0; a < DR_MINI; ++a)
#pragma unroll
                for (int b = 0; b <= a; ++b) {
                    // (row a starts at a (a - 1) / 2 among the keys' products and at a (a + 1) / 2 among the others)
                    const int vk = a * (a - 1) / 2 + b, vq = a * (a + 1) / 2 + b;
                    if (b < a) pk[vk < 0 ? 0 : vk] = fmaf(kr[a], kr[b], pk[vk < 0 ? 0 : vk]);
                    if (vq < 32) pq[vq & 31] = fmaf(qr[a], kr[b], pq[vq & 31]);
                    else px[(vq - 32) & 3] = fmaf(qr[a], kr[b], px[(vq - 32) & 3]);
                }
        }
#pragma unroll
        for (int v = 0; v < 4; ++v) pk[28 + v] = px[v];   // (the last four of the second kind fill up the first round)
        const float sk = dr_sums<4, false>(pk, lane), sq = dr_sums<4, false>(pq, lane);
        __syncwarp();
        if (lane < 28) kk[lane] = sk; else qk[32 + lane - 28] = sk;
        qk[lane] = sq;
        __syncwarp();
        for (int h0 = kvh * (H / G); h0 < (kvh + 1) * (H / G); h0 += 4) {   // four heads at a time, eight lanes each
            const int hs = lane >> 3, h = h0 + hs;
            const bool mine = h < (kvh + 1) * (H / G), there = mine && i < n;
            float g = 1.f, beta = 0.f;
            if (there) {
                g = expf(neg_exp_a[h] * dr_softplus(ab[(size_t)(t + i) * ldab + a_col + h] + dt_bias[h]));
                beta = 1.f / (1.f + expf(-ab[(size_t)(t + i) * ldab + b_col + h]));
            }
            float gs[DR_MINI], rho[DR_MINI], gamma = 1.f, after = 1.f;
#pragma unroll
            for (int j = 0; j < DR_MINI; ++j) gs[j] = __shfl_sync(0xffffffffu, g, j, 8);
#pragma unroll
            for (int j = DR_MINI - 1; j >= 0; --j) {   // rho[j]: the decays after j up to this token
                rho[j] = j >= i ? 1.f : rho[j + 1 < DR_MINI ? j + 1 : j] * gs[j + 1 < DR_MINI ? j + 1 : j];
                if (j > i) after *= gs[j]; else gamma *= gs[j];
            }
            float* A = a_s[warp][hs];
            __syncwarp();
#pragma unroll
            for (int j = 0; j < DR_MINI; ++j) A[i * 8 + j] = j < i ? beta * rho[j] * kk[i * (i - 1) / 2 + j] : 0.f;
            __syncwarp();
            float T[DR_MINI];   // column i of the inverse
#pragma unroll
            for (int a = 0; a < DR_MINI; ++a) {
                float s = a == i ? 1.f : 0.f;
#pragma unroll
                for (int l = 0; l < a; ++l) s = fmaf(-A[a * 8 + l], T[l], s);
                T[a] = a < i ? 0.f : s;
            }
            if (mine) {
                if (i < n) {
                    float* dst = coef + ((size_t)h * tokens + t + i) * DR_COEF;
                    *reinterpret_cast<float4*>(dst) = make_float4(beta, beta * gamma, gamma, after);
#pragma unroll
                    for (int j = 0; j < DR_MINI; ++j) dst[12 + j] = j <= i ? rho[j] * qk[i * (i + 1) / 2 + j] : 0.f;
                }
#pragma unroll
                for (int a = 0; a < DR_MINI; ++a)
                    if (a < n) coef[((size_t)h * tokens + t + a) * DR_COEF + 4 + i] = T[a];
            }
        }
        __syncwarp();
    }
}

// ---- the recurrence ----
// A block owns COLS columns of one head's state of one request, a warp CC of them (four, or two where there are few heads: then
// more warps share the SMs); lane l of the warp holds the rows RL l .. RL l + RL - 1 of its columns in registers, in pairs
// of rows (`fma.rn.f32x2`).  Per mini-chunk a lane forms its part of the products of eight keys and eight queries with the
// columns (in an order of the tokens of its own), the 8 CC of either kind are summed over the lanes together, and lane 8 c + i ends
// with those of token i and column c.
// u = (I + A)^-1 r is then eight products of numbers that the column's eight lanes exchange, and its multiples go through shared
// memory to all lanes for the update.  Tokens are staged DR_CHUNK at a time by bulk copies that one thread asks for, a chunk ahead.  Rows
// past D are zeros, tokens past a request's last have zero coefficients: they change nothing.
#define DR_CHUNK 16
#define DR_SMEM(DP, COLS) (sizeof(float) * (2 * DR_CHUNK * (2 * (DP) + (COLS) + DR_COEF) + 2 * DR_MINI * (COLS) * 2))
#define DR_SM_SMEM ((size_t)226 * 1024)   // what an SM's blocks share (a block's own limit is 227 KB with its static part)
#define DR_ERR_WALK 21

// Contiguous bytes from memory into shared memory, counted on an mbarrier (16-byte aligned, a multiple of 16 bytes).
__device__ __forceinline__ void dr_bulk(float* dst, const float* src, unsigned bytes, unsigned bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n"
                 ::"r"(tc_smem_u32(dst)), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

typedef unsigned long long dr_pair;   // two floats in a register pair
__device__ __forceinline__ dr_pair dr_pack(float lo, float hi) {
    dr_pair r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void dr_unpack(dr_pair v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ dr_pair dr_fma2(dr_pair a, dr_pair b, dr_pair c) {
    dr_pair r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ dr_pair dr_mul2(dr_pair a, dr_pair b) {
    dr_pair r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
// P pairs of floats from shared memory (8 P bytes, aligned to their number).
template <int P> __device__ __forceinline__ void dr_pairs(const float* p, dr_pair (&v)[P]) {
    if constexpr (P == 1) {
        v[0] = *reinterpret_cast<const dr_pair*>(p);
    } else {
#pragma unroll
        for (int e = 0; e < P; e += 2) {
            const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(p + 2 * e);
            v[e] = a.x;
            v[e + 1] = a.y;
        }
    }
}

template <int RL, int CC, int COLS>
__global__ void __launch_bounds__(COLS / CC * 32, 1)
delta_walk_kernel(const float* __restrict__ qk, const float* __restrict__ v, const float* __restrict__ coef, float* __restrict__ state,
                  float* __restrict__ ring, const void* __restrict__ x, int ldx, int x_bf16, const int* __restrict__ cu_seqlens,
                  const int* __restrict__ state_slots, const int* __restrict__ positions, float* __restrict__ out, int tokens, int G,
                  int D, int H, int Dv, int taps, int* __restrict__ error) {
    extern __shared__ __align__(16) float dr_smem[];
    __shared__ __align__(8) unsigned long long full_bar[2];
    __shared__ int failed;
    constexpr int DP = 32 * RL, P = RL / 2, THREADS = COLS / CC * 32, NV = 8 * CC;
    float* qk_s = dr_smem;                             // [2][DR_CHUNK][2][DP]
    float* v_s = qk_s + 2 * DR_CHUNK * 2 * DP;         // [2][COLS / 8][DR_CHUNK][8]
    float* c_s = v_s + 2 * DR_CHUNK * COLS;            // [2][DR_CHUNK][DR_COEF]
    float* u_s = c_s + 2 * DR_CHUNK * DR_COEF;         // [warps][2][DR_MINI][CC] twice each
    const int col0 = blockIdx.x * COLS, h = blockIdx.y, seq = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, ti = lane & 7, tc = (lane >> 3) & (CC - 1);
    const int kvh = h / (H / G), C = 2 * G * D + H * Dv, vblocks = (Dv + 7) >> 3;
    for (int i = threadIdx.x; i < 2 * DR_CHUNK * (2 * DP + COLS + DR_COEF); i += THREADS) dr_smem[i] = 0.f;
    if (threadIdx.x == 0) {
        tc_mbar_init(tc_smem_u32(&full_bar[0]), 1);
        tc_mbar_init(tc_smem_u32(&full_bar[1]), 1);
        failed = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");   // (the zeros before what the copies write)
    __syncthreads();
    pdl_wait();
    pdl_trigger();
    const int t0 = cu_seqlens[seq], t1 = cu_seqlens[seq + 1], slot = state_slots[seq];
    float* st = state + ((size_t)slot * H + h) * (size_t)Dv * D;

    // one thread asks for a chunk: the keys and queries, eight columns of values at a time, the coefficients
    auto stage = [&](int buf, int tb) {
        const int n = min(DR_CHUNK, t1 - tb), vb = min(COLS / 8, vblocks - col0 / 8);
        const unsigned bar = tc_smem_u32(&full_bar[buf]);
        tc_mbar_expect_tx(bar, (unsigned)(n * (2 * DP + vb * 8 + DR_COEF) * 4));
        dr_bulk(qk_s + buf * DR_CHUNK * 2 * DP, qk + ((size_t)kvh * tokens + tb) * 2 * DP, n * 2 * DP * 4, bar);
        for (int b = 0; b < vb; ++b)
            dr_bulk(v_s + (buf * (COLS / 8) + b) * DR_CHUNK * 8, v + (((size_t)h * vblocks + col0 / 8 + b) * tokens + tb) * 8, n * 32, bar);
        dr_bulk(c_s + buf * DR_CHUNK * DR_COEF, coef + ((size_t)h * tokens + tb) * DR_COEF, n * DR_COEF * 4, bar);
    };
    if (threadIdx.x == 0 && t1 > t0) stage(0, t0);
    dr_pair S[CC][P];
#pragma unroll
    for (int c = 0; c < CC; ++c) {
        const int col = col0 + warp * CC + c;
        float s[RL];
#pragma unroll
        for (int r = 0; r < RL; ++r) s[r] = col < Dv && RL * lane + r < D ? st[(size_t)col * D + RL * lane + r] : 0.f;
#pragma unroll
        for (int p = 0; p < P; ++p) S[c][p] = dr_pack(s[2 * p], s[2 * p + 1]);
    }
    int off[DR_MINI];   // where a lane's slot s finds its rows: token s xor (lane mod 8) of the mini-chunk
#pragma unroll
    for (int i = 0; i < DR_MINI; ++i) off[i] = (i ^ ti) * 2 * DP + RL * lane;
    int buf = 0, uses = 0;
    for (int tb = t0; tb < t1; tb += DR_CHUNK, buf ^= 1, ++uses) {
        const int n = min(DR_CHUNK, t1 - tb);
        if (!tc_mbar_wait(tc_smem_u32(&full_bar[buf]), (unsigned)((uses >> 1) & 1))) {
            failed = 1;
            atomicExch(error, DR_ERR_WALK);
        }
        // a request's last chunk: what an earlier one left in the rows past its end has coefficients too
        for (int i = n * DR_COEF + threadIdx.x; i < DR_CHUNK * DR_COEF; i += THREADS) c_s[buf * DR_CHUNK * DR_COEF + i] = 0.f;
        __syncthreads();   // (and everybody is done with the other buffer)
        if (failed) break;
        if (threadIdx.x == 0 && tb + DR_CHUNK < t1) stage(buf ^ 1, tb + DR_CHUNK);
        for (int m = 0; m < n; m += DR_MINI) {
            const float *qb = qk_s + (buf * DR_CHUNK + m) * 2 * DP, *kb = qb + DP;
            const float* cb = c_s + (buf * DR_CHUNK + m + ti) * DR_COEF;
            constexpr bool KEEP = RL <= 4;   // the keys stay in registers from the products to the update
            dr_pair kreg[KEEP ? DR_MINI : 1][P];
            float pk[NV], pq[NV];
#pragma unroll
            for (int i = 0; i < DR_MINI; ++i) {
                dr_pair k2[P];
                dr_pairs<P>(kb + off[i], k2);
#pragma unroll
                for (int e = 0; e < P; ++e)
                    if (KEEP) kreg[KEEP ? i : 0][e] = k2[e];
#pragma unroll
                for (int c = 0; c < CC; ++c) {
                    dr_pair a = dr_mul2(S[c][0], k2[0]);
#pragma unroll
                    for (int e = 1; e < P; ++e) a = dr_fma2(S[c][e], k2[e], a);
                    float lo, hi;
                    dr_unpack(a, lo, hi);
                    pk[c * 8 + i] = lo + hi;
                }
            }
            const float kS = dr_sums<CC, true>(pk, lane);
#pragma unroll
            for (int i = 0; i < DR_MINI; ++i) {
                dr_pair q2[P];
                dr_pairs<P>(qb + off[i], q2);
#pragma unroll
                for (int c = 0; c < CC; ++c) {
                    dr_pair a = dr_mul2(S[c][0], q2[0]);
#pragma unroll
                    for (int e = 1; e < P; ++e) a = dr_fma2(S[c][e], q2[e], a);
                    float lo, hi;
                    dr_unpack(a, lo, hi);
                    pq[c * 8 + i] = lo + hi;
                }
            }
            // lane 8 c + i: token m + i, column c of the warp
            const float4 c0 = *reinterpret_cast<const float4*>(cb);
            const float4 ta = *reinterpret_cast<const float4*>(cb + 4), tb4 = *reinterpret_cast<const float4*>(cb + 8);
            const float4 pa = *reinterpret_cast<const float4*>(cb + 12), pb4 = *reinterpret_cast<const float4*>(cb + 16);
            const float trow[8] = {ta.x, ta.y, ta.z, ta.w, tb4.x, tb4.y, tb4.z, tb4.w};
            const float prow[8] = {pa.x, pa.y, pa.z, pa.w, pb4.x, pb4.y, pb4.z, pb4.w};
            const int cl = warp * CC + tc;
            const float vt = v_s[((buf * (COLS / 8) + (cl >> 3)) * DR_CHUNK + m + ti) * 8 + (cl & 7)];
            const float r = fmaf(c0.x, vt, -c0.y * kS);
            float u0 = 0.f, u1 = 0.f;
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                u0 = fmaf(trow[j], __shfl_sync(0xffffffffu, r, j, 8), u0);
                u1 = fmaf(trow[j + 1], __shfl_sync(0xffffffffu, r, j + 1, 8), u1);
            }
            const float u = u0 + u1, wu = c0.w * u;
            float* us = u_s + (warp * 2 + ((m / DR_MINI) & 1)) * DR_MINI * 2 * CC;
            if (lane < NV) *reinterpret_cast<float2*>(us + (ti * CC + tc) * 2) = make_float2(wu, wu);
            // (token 0 of the mini-chunk is always there: its decay times those after it is the decay over the mini-chunk)
            const float gamma = __shfl_sync(0xffffffffu, c0.z * c0.w, 0, 8);
            const dr_pair gamma2 = dr_pack(gamma, gamma);
            __syncwarp();
#pragma unroll
            for (int c = 0; c < CC; ++c)
#pragma unroll
                for (int e = 0; e < P; ++e) S[c][e] = dr_mul2(S[c][e], gamma2);
#pragma unroll
            for (int i = 0; i < DR_MINI; ++i) {
                dr_pair w2[CC], k2[P];
                dr_pairs<CC>(us + (i ^ ti) * 2 * CC, w2);
                if (KEEP) {
#pragma unroll
                    for (int e = 0; e < P; ++e) k2[e] = kreg[KEEP ? i : 0][e];
                } else {
                    dr_pairs<P>(kb + off[i], k2);
                }
#pragma unroll
                for (int c = 0; c < CC; ++c)
#pragma unroll
                    for (int e = 0; e < P; ++e) S[c][e] = dr_fma2(k2[e], w2[c], S[c][e]);
            }
            const float qS = dr_sums<CC, true>(pq, lane);
            float o0 = c0.z * qS, o1 = 0.f;
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                o0 = fmaf(prow[j], __shfl_sync(0xffffffffu, u, j, 8), o0);
                o1 = fmaf(prow[j + 1], __shfl_sync(0xffffffffu, u, j + 1, 8), o1);
            }
            const int col = col0 + warp * CC + tc;
            if (lane < NV && m + ti < n && col < Dv) out[((size_t)(tb + m + ti) * H + h) * Dv + col] = o0 + o1;
        }
    }
#pragma unroll
    for (int c = 0; c < CC; ++c) {
        const int col = col0 + warp * CC + c;
#pragma unroll
        for (int p = 0; p < P; ++p) {
            float lo, hi;
            dr_unpack(S[c][p], lo, hi);
            const int d = RL * lane + 2 * p;
            if (col < Dv && d < D) st[(size_t)col * D + d] = lo;
            if (col < Dv && d + 1 < D) st[(size_t)col * D + d + 1] = hi;
        }
    }
    // the request's last inputs of the convolutions, its blocks sharing the channels
    const int part = blockIdx.y * gridDim.x + blockIdx.x, parts = gridDim.x * gridDim.y;
    for (int c = part * THREADS + threadIdx.x; c < C; c += parts * THREADS)
        for (int t = max(t0, t1 - (taps - 1)); t < t1; ++t)
            ring[((size_t)slot * taps + positions[t] % taps) * C + c] =
                x_bf16 ? to_f32(((const bf16*)x)[(size_t)t * ldx + c]) : ((const float*)x)[(size_t)t * ldx + c];
}

// neg_exp_a, dt_bias float32 [H]: -exp(A_log) and the decay's offset.  ab float32 [tokens, ldab]: a and b of head h in columns
// a_col + h, b_col + h.  qk: from `vx_delta_conv` of the same step.  coef float32 [H, tokens, 20], 16-byte aligned.
extern "C" int vx_delta_coef(const float* qk, const float* ab, int ldab, int a_col, int b_col, const float* neg_exp_a,
                             const float* dt_bias, const int* seq_of_token, const int* cu_seqlens, float* coef, int tokens, int G, int D,
                             int H, int Dv, cudaStream_t stream) {
    if (tokens <= 0) return VX_OK;
    if (G <= 0 || D <= 0 || H <= 0 || Dv <= 0 || H % G || ldab < a_col + H || ldab < b_col + H || a_col < 0 || b_col < 0) return VX_ERR_SHAPE;
    if (((uintptr_t)coef) & 15) return VX_ERR_ALIGN;
    const long long warps = (long long)((tokens + DR_MINI - 1) / DR_MINI) * G;
    if (warps / DR_CW > 0x7ffffff0LL) return VX_ERR_LIMIT;
    VX_LAUNCH_K(VX_K_ELEMENTWISE, delta_coef_kernel, (unsigned)((warps + DR_CW - 1) / DR_CW), DR_CW * 32, 0, stream, qk, ab, ldab, a_col,
                b_col, neg_exp_a, dt_bias, seq_of_token, cu_seqlens, coef, tokens, G, D, H);
    VX_LAUNCH_CHECK();
    return VX_OK;
}

// qk, v, coef: from the two entries above; x, ldx: what `vx_delta_conv` read.  state float32 [slots, H, Dv, D], ring float32
// [slots, taps, C]: read and written.  out float32 [tokens, H * Dv].  layout: warps of two columns in blocks of 8 (1),
// warps of four in blocks of 16 (2), or 0 for the kernel's choice.  `error`: a device int that a block sets if its wait
// for its own copies runs out.
extern "C" int vx_delta_walk(const float* qk, const float* v, const float* coef, float* state, float* ring, const void* x, int ldx,
                             const int* cu_seqlens, const int* state_slots, const int* positions, float* out, int tokens, int seqs, int G,
                             int D, int H, int Dv, int taps, int layout, int* error, int dtype, cudaStream_t stream) {
    if (seqs <= 0) return VX_OK;
    if (G <= 0 || D <= 0 || H <= 0 || Dv <= 0 || H % G || taps <= 0 || ldx < 2 * G * D + H * Dv) return VX_ERR_SHAPE;
    if (D > 256 || taps > DR_MAX_TAPS || seqs > 65535 || H > 65535) return VX_ERR_LIMIT;
    if (dtype != VX_F32 && dtype != VX_BF16) return VX_ERR_DTYPE;
    if (((uintptr_t)qk | (uintptr_t)v | (uintptr_t)coef) & 15) return VX_ERR_ALIGN;
    if (!error || tokens <= 0) return VX_ERR_SHAPE;
    static bool configured[6][VX_MAX_DEVICES];
    static int sms[VX_MAX_DEVICES];
    // few heads: warps of two columns, blocks of 8; many: warps of four, blocks of 16 (a column's sums do not depend on it)
    const long long units = (long long)H * seqs * ((Dv + 7) / 8);
    if (!layout) layout = D <= 128 && units <= 2LL * vx_sm_count(sms) ? 1 : 2;
    if (layout < 0 || layout > 2) return VX_ERR_SHAPE;
    const int cols = layout == 1 ? 8 : 16;
    dim3 grid((Dv + cols - 1) / cols, H, seqs);
    // as much shared memory a block as lets no SM take more blocks than its share: these blocks become resident while the kernel
    // before them still runs, and would crowd on the SMs that are free first
    const long long share = ((long long)grid.x * grid.y * grid.z + vx_sm_count(sms) - 1) / vx_sm_count(sms);
    const size_t spread = share <= 4 ? DR_SM_SMEM / share - 2048 : 0;
#define DR_GO(RL_, CC_, COLS_, SLOT)                                                                                            \
    do {                                                                                                                        \
        if (int rc = vx_configure_smem(delta_walk_kernel<RL_, CC_, COLS_>, DR_SM_SMEM, configured[SLOT])) return rc;           \
        const size_t need = DR_SMEM(32 * RL_, COLS_);                                                                           \
        VX_LAUNCH_K(VX_K_ATTENTION, (delta_walk_kernel<RL_, CC_, COLS_>), grid, COLS_ / CC_ * 32, need > spread ? need : spread, stream, \
                    qk, v, coef, state, ring, x, ldx, dtype == VX_BF16 ? 1 : 0, cu_seqlens, state_slots, positions, out, tokens, G, \
                    D, H, Dv, taps, error);                                                                                    \
    } while (0)
#define DR_GO_CC(RL_, SLOT)                                                                                                    \
    do {                                                                                                                       \
        if (layout == 1) DR_GO(RL_, 2, 8, SLOT); else DR_GO(RL_, 4, 16, SLOT + 1);                                             \
    } while (0)
    if (D <= 64) DR_GO_CC(2, 0);
    else if (D <= 128) DR_GO_CC(4, 2);
    else DR_GO_CC(8, 4);
#undef DR_GO_CC
#undef DR_GO
    VX_LAUNCH_CHECK();
    return VX_OK;
}

// ---- a step of single tokens ----
// One block per (head, request): row t of the step is request t's only token.  Eight lanes a column of the state as in the
// walk, all of a head's columns in the block (128 at a time).  The state, the ring and the step's description are older than
// the kernel right before this one (the projections), so they are read before the wait for it.  The norms' sums and q . k are
// formed beside the products with the state.  Then every head's o / sqrt(mean(o^2) + eps) * norm * silu(gate).
template <typename TX, typename T, int R>
__global__ void __launch_bounds__(1024)
delta_decode_kernel(const TX* __restrict__ x, int ldx, int g_col, const float* __restrict__ ab, int ldab, int a_col, int b_col,
                    const float* __restrict__ w, const float* __restrict__ neg_exp_a, const float* __restrict__ dt_bias,
                    const float* __restrict__ norm_w, float* __restrict__ state, float* __restrict__ ring,
                    const int* __restrict__ state_slots, const int* __restrict__ positions, T* __restrict__ out, int G, int D, int H,
                    int Dv, int taps, float q_mul, float eps) {
    extern __shared__ __align__(16) float dr_smem[];
    __shared__ float scratch[32];
    constexpr int DP = 8 * R;
    float *q_s = dr_smem, *k_s = q_s + DP, *v_s = k_s + DP, *o_s = v_s + Dv;
    const int h = blockIdx.x, t = blockIdx.y, group = H / G, kvh = h / group, C = 2 * G * D + H * Dv;
    const int li = threadIdx.x & 7, pass_cols = blockDim.x >> 3;
    const int slot = state_slots[t], pos = positions[t];
    float* rg = ring + (size_t)slot * taps * C;
    float* st0 = state + ((size_t)slot * H + h) * (size_t)Dv * D;
    float S[R];
    auto load_state = [&](int col) {
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
            const int d = 4 * li + 32 * j;
            if (col < Dv && d < D && (D & 3) == 0) {
                const float4 s4 = *reinterpret_cast<const float4*>(st0 + (size_t)col * D + d);
                S[4 * j] = s4.x; S[4 * j + 1] = s4.y; S[4 * j + 2] = s4.z; S[4 * j + 3] = s4.w;
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) S[4 * j + e] = col < Dv && d + e < D ? st0[(size_t)col * D + d + e] : 0.f;
            }
        }
    };
    load_state(threadIdx.x >> 3);
    auto channel = [&](int i) { return i < D ? kvh * D + i : (i < 2 * D ? G * D + kvh * D + i - D : 2 * G * D + h * Dv + i - 2 * D); };
    auto earlier = [&](int c) {   // the convolution's part that the ring holds
        float s = 0.f;
        for (int j = min(taps - 1, pos); j > 0; --j) s = fmaf(w[(size_t)(taps - 1 - j) * C + c], rg[(size_t)((pos - j) % taps) * C + c], s);
        return s;
    };
    const int all = 2 * D + Dv;
    const float first = (int)threadIdx.x < all ? earlier(channel(threadIdx.x)) : 0.f;
    for (int i = D + threadIdx.x; i < DP; i += blockDim.x) { q_s[i] = 0.f; k_s[i] = 0.f; }
    const float neg_a = neg_exp_a[h], bias = dt_bias[h];
    pdl_wait();
    pdl_trigger();
    const TX* row = x + (size_t)t * ldx;
    for (int i = threadIdx.x; i < all; i += blockDim.x) {
        const int c = channel(i);
        const float xv = to_f32(row[c]);
        const float s = dr_silu(fmaf(w[(size_t)(taps - 1) * C + c], xv, i < (int)blockDim.x ? first : earlier(c)));
        (i < D ? q_s[i] : (i < 2 * D ? k_s[i - D] : v_s[i - 2 * D])) = s;
        // (row pos mod taps: none of those that `earlier` reads, whatever the order of the heads that share q and k)
        if (taps > 1 && (i >= 2 * D || h == kvh * group)) rg[(size_t)(pos % taps) * C + c] = xv;
    }
    const float g = expf(neg_a * dr_softplus(ab[(size_t)t * ldab + a_col + h] + bias));
    const float beta = 1.f / (1.f + expf(-ab[(size_t)t * ldab + b_col + h]));
    __syncthreads();
    for (int col = threadIdx.x >> 3; col < ((Dv + 3) & ~3); col += pass_cols) {   // (whole warps: 4 columns each)
        if (col >= pass_cols) load_state(col);
        float kS = 0.f, qS = 0.f, kk = 0.f, qq = 0.f, qk = 0.f;
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
            const float4 k4 = *reinterpret_cast<const float4*>(k_s + 4 * li + 32 * j);
            const float4 q4 = *reinterpret_cast<const float4*>(q_s + 4 * li + 32 * j);
            const float kv[4] = {k4.x, k4.y, k4.z, k4.w}, qv[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                kS = fmaf(S[4 * j + e], kv[e], kS);
                qS = fmaf(S[4 * j + e], qv[e], qS);
                kk = fmaf(kv[e], kv[e], kk);
                qq = fmaf(qv[e], qv[e], qq);
                qk = fmaf(qv[e], kv[e], qk);
            }
        }
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) {
            kS += __shfl_xor_sync(0xffffffffu, kS, o);
            qS += __shfl_xor_sync(0xffffffffu, qS, o);
            kk += __shfl_xor_sync(0xffffffffu, kk, o);
            qq += __shfl_xor_sync(0xffffffffu, qq, o);
            qk += __shfl_xor_sync(0xffffffffu, qk, o);
        }
        const float kn = rsqrtf(kk + DR_EPS_UNIT), qn = rsqrtf(qq + DR_EPS_UNIT) * q_mul;
        const float u = beta * ((col < Dv ? v_s[col] : 0.f) - g * kn * kS);
        if (li == 0 && col < Dv) o_s[col] = qn * fmaf(kn * qk, u, g * qS);
        const float ku = kn * u;
        if (col < Dv) {
#pragma unroll
            for (int j = 0; j < R / 4; ++j) {
                const int d = 4 * li + 32 * j;
                if (d >= D) continue;
                const float4 k4 = *reinterpret_cast<const float4*>(k_s + d);
                const float4 n4 = make_float4(fmaf(k4.x, ku, g * S[4 * j]), fmaf(k4.y, ku, g * S[4 * j + 1]),
                                              fmaf(k4.z, ku, g * S[4 * j + 2]), fmaf(k4.w, ku, g * S[4 * j + 3]));
                float* dst = st0 + (size_t)col * D + d;
                if ((D & 3) == 0) {
                    *reinterpret_cast<float4*>(dst) = n4;
                } else {
                    const float nv[4] = {n4.x, n4.y, n4.z, n4.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        if (d + e < D) dst[e] = nv[e];
                }
            }
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int i = threadIdx.x; i < Dv; i += blockDim.x) ss = fmaf(o_s[i], o_s[i], ss);
    ss = block_sum(ss, scratch);
    const float rstd = rsqrtf(ss / (float)Dv + eps);
    for (int i = threadIdx.x; i < Dv; i += blockDim.x)
        out[((size_t)t * H + h) * Dv + i] = from_f32<T>(o_s[i] * rstd * norm_w[i] * dr_silu(to_f32(row[g_col + (size_t)h * Dv + i])));
}

template <typename TX, typename T>
static int launch_delta_decode(const TX* x, int ldx, int g_col, const float* ab, int ldab, int a_col, int b_col, const float* w,
                               const float* neg_exp_a, const float* dt_bias, const float* norm_w, float* state, float* ring,
                               const int* state_slots, const int* positions, T* out, int requests, int G, int D, int H, int Dv, int taps,
                               float q_mul, float eps, cudaStream_t stream) {
    int threads = (8 * Dv + 31) & ~31;
    if (threads > 1024) threads = 1024;
#define DR_GO(R_)                                                                                                               \
    VX_LAUNCH_K(VX_K_ATTENTION, (delta_decode_kernel<TX, T, R_>), dim3(H, requests), threads, (2 * 8 * R_ + 2 * Dv) * sizeof(float), \
                stream, x, ldx, g_col, ab, ldab, a_col, b_col, w, neg_exp_a, dt_bias, norm_w, state, ring, state_slots, positions,   \
                out, G, D, H, Dv, taps, q_mul, eps)
    if (D <= 32) DR_GO(4);
    else if (D <= 64) DR_GO(8);
    else if (D <= 128) DR_GO(16);
    else DR_GO(32);
#undef DR_GO
    VX_LAUNCH_CHECK();
    return VX_OK;
}

// x [requests, ldx]: q, k, v from column 0 on and the gates [H, Dv] at column g_col, in x_dtype (float32 with outputs of either
// type, or the outputs' own); the rest as in the two entries above.  out [requests, H * Dv] in `dtype`.
extern "C" int vx_delta_decode(const void* x, int ldx, int g_col, const float* ab, int ldab, int a_col, int b_col, const float* w,
                               const float* neg_exp_a, const float* dt_bias, const float* norm_w, float* state, float* ring,
                               const int* state_slots, const int* positions, void* out, int requests, int G, int D, int H, int Dv,
                               int taps, float q_mul, float eps, int x_dtype, int dtype, cudaStream_t stream) {
    if (requests <= 0) return VX_OK;
    if (G <= 0 || D <= 0 || H <= 0 || Dv <= 0 || H % G || taps <= 0 || g_col < 2 * G * D + H * Dv || ldx < g_col + H * Dv) return VX_ERR_SHAPE;
    if (ldab < a_col + H || ldab < b_col + H || a_col < 0 || b_col < 0) return VX_ERR_SHAPE;
    if (D > 256 || Dv > 4096 || taps > DR_MAX_TAPS || requests > 65535) return VX_ERR_LIMIT;
#define DR_GO(TX_, T_)                                                                                                          \
    launch_delta_decode<TX_, T_>((const TX_*)x, ldx, g_col, ab, ldab, a_col, b_col, w, neg_exp_a, dt_bias, norm_w, state, ring, state_slots, \
                                 positions, (T_*)out, requests, G, D, H, Dv, taps, q_mul, eps, stream)
    if (x_dtype == VX_F32 && dtype == VX_F32) return DR_GO(float, float);
    if (x_dtype == VX_F32 && dtype == VX_BF16) return DR_GO(float, bf16);
    if (x_dtype == VX_BF16 && dtype == VX_BF16) return DR_GO(bf16, bf16);
#undef DR_GO
    return VX_ERR_DTYPE;
}
