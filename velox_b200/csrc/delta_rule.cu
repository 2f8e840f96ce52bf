// The gated delta rule: per head a state S [D, Dv] that forgets, and that a token corrects instead of adding to:
//   S' = g_t S_(t-1);  u_t = beta_t (v_t - S'^T k_t);  S_t = S' + k_t u_t^T;  o_t = S_t^T q_t
// with q, k, v behind a short causal convolution over time (per channel, then silu), q and k unit vectors per head, a decay
// g = exp(-exp(A_log) softplus(a + dt_bias)) and a step size beta = sigmoid(b) per head and token.  Several heads may share
// one q/k head.
//
//   delta_conv      convolution, silu and unit vectors of a step's tokens (float32 out), and every key's products with the
//                   keys and queries near it
//   delta_walk      the recurrence over a step's tokens; afterwards the last inputs of the convolutions go into their slots
//   delta_decode    a step of single tokens: both of these, the norm of every head's output and its gate in one kernel
//
// State per request (float32): S transposed, [H, Dv, D] (a column of S is contiguous), and the last inputs of the
// convolutions as a ring [taps, channels]: position p lies in row p mod taps.  A token at position p reads rows p - 1 ..
// p - taps + 1 and writes row p, which is none of those, so the blocks of a decode step need no order among them.  Rows of
// positions before 0 count as zeros and are never read.  Channels are numbered q [G, D], k [G, D], v [H, Dv].
#include "mma_helpers.cuh"

#define DR_EPS_UNIT 1e-6f
#define DR_DOTS 8      // per token and q/k head: k.k of the tokens 1, 2, 3 back (0 .. 2), q.k of itself and 1, 2, 3 back (3 .. 6)
#define DR_MINI 4      // tokens of a mini-chunk
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
// y float32 [tokens, C] with C = 2 G D + H Dv: q as a unit vector times q_mul, k as a unit vector, v.  dots float32
// [tokens, G, DR_DOTS], where the tokens it reaches back to lie among the rows that the request brings (else whatever).
// A warp takes one unit (the q and k of one head, or a run of v's channels) of one token.  Any sizes (D up to 256).
template <typename T>
__device__ __forceinline__ float dr_conv_at(const T* __restrict__ x, int ldx, const float* __restrict__ w, int C, int taps, int t,
                                            const DrPlace& at, int c) {
    float s = 0.f;
    for (int j = taps - 1; j >= 0; --j) {
        float v = 0.f;
        if (at.local >= j) v = to_f32(x[(size_t)(t - j) * ldx + c]);
        else if (at.pos >= j) v = at.ring[(size_t)((at.pos - j) % taps) * C + c];
        s = fmaf(w[(size_t)(taps - 1 - j) * C + c], v, s);
    }
    return dr_silu(s);
}

template <typename T>
__global__ void __launch_bounds__(128)
delta_conv_any_kernel(const T* __restrict__ x, int ldx, const float* __restrict__ w, const float* __restrict__ ring,
                      const int* __restrict__ seq_of_token, const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots,
                      const int* __restrict__ positions, float* __restrict__ y, float* __restrict__ dots, int tokens, int G, int D,
                      int HDv, int taps, float q_mul, int units) {
    pdl_wait();
    pdl_trigger();
    const long long id = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    const int t = (int)(id / units), unit = (int)(id - (long long)t * units);
    if (t >= tokens) return;
    const int C = 2 * G * D + HDv;
    const DrPlace at = dr_place(t, seq_of_token, cu_seqlens, state_slots, positions, ring, (size_t)taps * C);
    float* yr = y + (size_t)t * C;
    if (unit >= G) {   // 256 channels of v
        const int c0 = 2 * G * D + (unit - G) * 256;
        for (int i = lane; i < 256 && c0 + i < C; i += 32) yr[c0 + i] = dr_conv_at(x, ldx, w, C, taps, t, at, c0 + i);
        return;
    }
    const int qc = unit * D, kc = G * D + unit * D;
    float q[8], k[DR_MINI][8], kn[DR_MINI], qn = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int d = lane + 32 * i;
        q[i] = d < D ? dr_conv_at(x, ldx, w, C, taps, t, at, qc + d) : 0.f;
        qn = fmaf(q[i], q[i], qn);
    }
    qn = rsqrtf(warp_sum(qn) + DR_EPS_UNIT) * q_mul;
#pragma unroll
    for (int b = 0; b < DR_MINI; ++b) {   // the token's key and those of the three before it
        float ss = 0.f;
        const bool there = at.local >= b;
        const DrPlace ab{at.local - b, at.pos - b, at.ring};
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int d = lane + 32 * i;
            k[b][i] = d < D && there ? dr_conv_at(x, ldx, w, C, taps, t - b, ab, kc + d) : 0.f;
            ss = fmaf(k[b][i], k[b][i], ss);
        }
        kn[b] = rsqrtf(warp_sum(ss) + DR_EPS_UNIT);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int d = lane + 32 * i;
        if (d < D) {
            yr[qc + d] = q[i] * qn;
            yr[kc + d] = k[0][i] * kn[0];
        }
    }
    float* dr = dots + ((size_t)t * G + unit) * DR_DOTS;
#pragma unroll
    for (int b = 0; b < DR_MINI; ++b) {
        float kk = 0.f, qk = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            kk = fmaf(k[0][i], k[b][i], kk);
            qk = fmaf(q[i], k[b][i], qk);
        }
        kk = warp_sum(kk) * kn[0] * kn[b];
        qk = warp_sum(qk) * qn * kn[b];
        if (lane == 0) {
            if (b) dr[b - 1] = kk;
            dr[3 + b] = qk;
        }
    }
}

// The same for four taps and heads of 32 VEC channels, a warp taking RUN consecutive tokens of a unit: every row it needs
// is asked for before the first is used and read once, not once a tap.
#define DR_RUN 8
template <typename T, int VEC>
__global__ void __launch_bounds__(128)
delta_conv_run_kernel(const T* __restrict__ x, int ldx, const float* __restrict__ w, const float* __restrict__ ring,
                      const int* __restrict__ seq_of_token, const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots,
                      const int* __restrict__ positions, float* __restrict__ y, float* __restrict__ dots, int tokens, int G, int HDv,
                      float q_mul, int units) {
    constexpr int TAPS = 4, D = 32 * VEC, BACK = DR_MINI - 1;
    const int C = 2 * G * D + HDv;
    const int lane = threadIdx.x & 31;
    const long long id = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    const int unit = (int)(id % units), t0 = (int)(id / units) * DR_RUN;
    if (t0 >= tokens) {   // (a warp past the end; the block's first warp never is)
        return;
    }
    const bool is_v = unit >= G;
    const int c = is_v ? 2 * G * D + (unit - G) * D + lane * VEC : unit * D + lane * VEC;   // v's or q's channel
    const bool live = c < C;
    float wt[TAPS][VEC];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) wt[j][e] = 0.f;
        if (live) dr_load<VEC>(w + (size_t)j * C + c, wt[j]);
    }
    pdl_wait();
    pdl_trigger();
    // the convolution of token t from those of the rows win[first + TAPS - 1 - j] = x[t - j] that its request brings
    auto conv = [&](const auto& win, int first, const float (&wk)[TAPS][VEC], int t, int ch, float (&out)[VEC]) {
        const DrPlace at = dr_place(t, seq_of_token, cu_seqlens, state_slots, positions, ring, (size_t)TAPS * C);
#pragma unroll
        for (int e = 0; e < VEC; ++e) out[e] = 0.f;
#pragma unroll
        for (int j = TAPS - 1; j >= 0; --j) {
            float v[VEC];
            if (at.local >= j) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) v[e] = win[first + TAPS - 1 - j][e];
            } else if (at.pos >= j && ch < C) {
                dr_load<VEC>(at.ring + (size_t)((at.pos - j) % TAPS) * C + ch, v);
            } else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) v[e] = 0.f;
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) out[e] = fmaf(wk[TAPS - 1 - j][e], v[e], out[e]);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) out[e] = dr_silu(out[e]);
    };
    auto row = [&](int r, int ch, float (&v)[VEC]) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = 0.f;
        if (r >= 0 && r < tokens && ch < C) dr_load<VEC>(x + (size_t)r * ldx + ch, v);
    };
    if (is_v) {
        float win[DR_RUN + TAPS - 1][VEC];
#pragma unroll
        for (int i = 0; i < DR_RUN + TAPS - 1; ++i) row(t0 - (TAPS - 1) + i, c, win[i]);
#pragma unroll
        for (int u = 0; u < DR_RUN; ++u) {
            const int t = t0 + u;
            if (t >= tokens) break;
            float o[VEC];
            conv(win, u, wt, t, c, o);
            if (live) dr_store<VEC>(y + (size_t)t * C + c, o);
        }
        return;
    }
    const int ck = G * D + c;
    float wk[TAPS][VEC];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) dr_load<VEC>(w + (size_t)j * C + ck, wk[j]);
    float qw[DR_RUN + TAPS - 1][VEC], kw[DR_RUN + BACK + TAPS - 1][VEC];
#pragma unroll
    for (int i = 0; i < DR_RUN + BACK + TAPS - 1; ++i) row(t0 - BACK - (TAPS - 1) + i, ck, kw[i]);
#pragma unroll
    for (int i = 0; i < DR_RUN + TAPS - 1; ++i) row(t0 - (TAPS - 1) + i, c, qw[i]);
    float kh[DR_MINI][VEC];   // unit keys: [b] of the token b back
#pragma unroll
    for (int b = 0; b < DR_MINI; ++b)
#pragma unroll
        for (int e = 0; e < VEC; ++e) kh[b][e] = 0.f;
#pragma unroll
    for (int u = -BACK; u < DR_RUN; ++u) {
        const int t = t0 + u;
        if (t >= tokens) break;
#pragma unroll
        for (int b = DR_MINI - 1; b > 0; --b)
#pragma unroll
            for (int e = 0; e < VEC; ++e) kh[b][e] = kh[b - 1][e];
        if (t < 0) continue;
        conv(kw, u + BACK, wk, t, ck, kh[0]);
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss = fmaf(kh[0][e], kh[0][e], ss);
        const float kn = rsqrtf(warp_sum(ss) + DR_EPS_UNIT);
#pragma unroll
        for (int e = 0; e < VEC; ++e) kh[0][e] *= kn;
        if (u < 0) continue;
        float q[VEC];
        conv(qw, u, wt, t, c, q);
        ss = 0.f;
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss = fmaf(q[e], q[e], ss);
        const float qn = rsqrtf(warp_sum(ss) + DR_EPS_UNIT) * q_mul;
#pragma unroll
        for (int e = 0; e < VEC; ++e) q[e] *= qn;
        dr_store<VEC>(y + (size_t)t * C + c, q);
        dr_store<VEC>(y + (size_t)t * C + ck, kh[0]);
        float p[DR_DOTS];
#pragma unroll
        for (int b = 0; b < DR_DOTS; ++b) p[b] = 0.f;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
#pragma unroll
            for (int b = 1; b < DR_MINI; ++b) p[b - 1] = fmaf(kh[0][e], kh[b][e], p[b - 1]);
#pragma unroll
            for (int b = 0; b < DR_MINI; ++b) p[3 + b] = fmaf(q[e], kh[b][e], p[3 + b]);
        }
        // eight sums over 32 lanes: halves of the values change sides, so lane l ends with the sum number (l >> 2)
        float a4[4], a2[2], a1;
        const bool h16 = lane & 16, h8 = lane & 8, h4 = lane & 4;
#pragma unroll
        for (int i = 0; i < 4; ++i) a4[i] = (h16 ? p[4 + i] : p[i]) + __shfl_xor_sync(0xffffffffu, h16 ? p[i] : p[4 + i], 16);
#pragma unroll
        for (int i = 0; i < 2; ++i) a2[i] = (h8 ? a4[2 + i] : a4[i]) + __shfl_xor_sync(0xffffffffu, h8 ? a4[i] : a4[2 + i], 8);
        a1 = (h4 ? a2[1] : a2[0]) + __shfl_xor_sync(0xffffffffu, h4 ? a2[0] : a2[1], 4);
        a1 += __shfl_xor_sync(0xffffffffu, a1, 2);
        a1 += __shfl_xor_sync(0xffffffffu, a1, 1);
        if ((lane & 3) == 0) dots[((size_t)t * G + unit) * DR_DOTS + (lane >> 2)] = a1;
    }
}

template <typename T>
static int launch_delta_conv(const T* x, int ldx, const float* w, const float* ring, const int* seq_of_token, const int* cu_seqlens,
                             const int* state_slots, const int* positions, float* y, float* dots, int tokens, int G, int D, int H,
                             int Dv, int taps, float q_mul, cudaStream_t stream) {
    const int HDv = H * Dv, vec = D / 32, C = 2 * G * D + HDv;
    const bool run = taps == 4 && (D == 32 || D == 64 || D == 128) && tokens > 1 && HDv % vec == 0 && ldx % vec == 0 &&
                     !(((uintptr_t)x | (uintptr_t)w | (uintptr_t)ring | (uintptr_t)y) & 15) && C % vec == 0;
    const int units = G + (run ? (HDv + D - 1) / D : (HDv + 255) / 256);
    const long long warps = (long long)units * (run ? (tokens + DR_RUN - 1) / DR_RUN : tokens);
    if ((warps + 3) / 4 > 0x7fffffffLL) return VX_ERR_LIMIT;
    const unsigned blocks = (unsigned)((warps + 3) / 4);
#define DR_GO(V_) VX_LAUNCH_K(VX_K_ELEMENTWISE, (delta_conv_run_kernel<T, V_>), blocks, 128, 0, stream, x, ldx, w, ring, seq_of_token, \
                              cu_seqlens, state_slots, positions, y, dots, tokens, G, HDv, q_mul, units)
    if (run && vec == 1) DR_GO(1);
    else if (run && vec == 2) DR_GO(2);
    else if (run) DR_GO(4);
    else
        VX_LAUNCH_K(VX_K_ELEMENTWISE, (delta_conv_any_kernel<T>), blocks, 128, 0, stream, x, ldx, w, ring, seq_of_token, cu_seqlens,
                    state_slots, positions, y, dots, tokens, G, D, HDv, taps, q_mul, units);
#undef DR_GO
    VX_LAUNCH_CHECK();
    return VX_OK;
}

// x [tokens, ldx]: the projections q [G, D], k [G, D], v [H, Dv] from column 0 on.  w float32 [taps, C] (the last row is the
// current token's), ring float32 [slots, taps, C] (read only).  y, dots: see `delta_conv_any_kernel`.
extern "C" int vx_delta_conv(const void* x, int ldx, const float* w, const float* ring, const int* seq_of_token,
                             const int* cu_seqlens, const int* state_slots, const int* positions, float* y, float* dots, int tokens,
                             int G, int D, int H, int Dv, int taps, float q_mul, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return VX_OK;
    if (G <= 0 || D <= 0 || H <= 0 || Dv <= 0 || H % G || taps <= 0 || ldx < 2 * G * D + H * Dv) return VX_ERR_SHAPE;
    if (D > 256 || taps > DR_MAX_TAPS) return VX_ERR_LIMIT;
    if (dtype == VX_F32)
        return launch_delta_conv<float>((const float*)x, ldx, w, ring, seq_of_token, cu_seqlens, state_slots, positions, y, dots, tokens,
                                        G, D, H, Dv, taps, q_mul, stream);
    if (dtype == VX_BF16)
        return launch_delta_conv<bf16>((const bf16*)x, ldx, w, ring, seq_of_token, cu_seqlens, state_slots, positions, y, dots, tokens,
                                       G, D, H, Dv, taps, q_mul, stream);
    return VX_ERR_DTYPE;
}

// ---- the recurrence ----
// A block owns DR_COLS columns of one head's state of one request, a warp four of them, eight lanes a column: lane i of the
// eight holds the rows 4 i + 32 j .. + 3 (R of them) in registers.  Tokens are taken DR_MINI at a time.  With gamma_i the
// product of the decays up to token i of the mini-chunk and rho_ij that of the decays after j up to i, the rule unrolls to
//   u_i = beta_i (v_i - gamma_i (k_i . S) - sum_(j < i) rho_ij (k_i . k_j) u_j)
//   o_i = gamma_i (q_i . S) + sum_(j <= i) rho_ij (q_i . k_j) u_j
//   S  <- gamma_3 S + sum_j rho_3j k_j u_j^T
// with S the state before the mini-chunk: the eight products with S of a mini-chunk do not wait for one another, and are
// summed over the eight lanes together.  The products among keys and queries come from `delta_conv`.  Tokens are staged
// DR_CHUNK at a time by asynchronous copies, a chunk ahead; their coefficients (three float4 a token) likewise, by a warp in
// turn.  Tokens past a request's last count as k = q = v = 0, beta = 0, g = 1, which changes nothing.
#define DR_WARPS 4
#define DR_COLS (DR_WARPS * 4)
#define DR_CHUNK 16
#define DR_COEF 12
#define DR_SMEM(DP) (sizeof(float) * 2 * DR_CHUNK * (2 * (DP) + DR_COLS + DR_COEF))

__device__ __forceinline__ void dr_copy4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

struct DrGates {   // what a token's coefficients are made from
    float a, b, kk[3], qk[4];
};

template <int R>
__global__ void __launch_bounds__(DR_WARPS * 32)
delta_walk_kernel(const float* __restrict__ y, const float* __restrict__ dots, const float* __restrict__ ab, int ldab, int a_col,
                  int b_col, const float* __restrict__ neg_exp_a, const float* __restrict__ dt_bias, float* __restrict__ state,
                  float* __restrict__ ring, const void* __restrict__ x, int ldx, int x_bf16, const int* __restrict__ cu_seqlens,
                  const int* __restrict__ state_slots, const int* __restrict__ positions, float* __restrict__ out, int G, int D,
                  int H, int Dv, int taps) {
    extern __shared__ __align__(16) float dr_smem[];
    constexpr int DP = 8 * R;
    float* q_s = dr_smem;                              // [2][DR_CHUNK][DP]
    float* k_s = q_s + 2 * DR_CHUNK * DP;              // [2][DR_CHUNK][DP]
    float* v_s = k_s + 2 * DR_CHUNK * DP;              // [2][DR_CHUNK][DR_COLS]
    float* c_s = v_s + 2 * DR_CHUNK * DR_COLS;         // [2][DR_CHUNK][DR_COEF]
    const int col0 = blockIdx.x * DR_COLS, h = blockIdx.y, seq = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, li = lane & 7;
    const int kvh = h / (H / G), C = 2 * G * D + H * Dv;
    const int cl = warp * 4 + (lane >> 3), col = col0 + cl;
    const float neg_a = neg_exp_a[h], bias = dt_bias[h];
    for (int i = threadIdx.x; i < 2 * DR_CHUNK * (2 * DP + DR_COLS); i += DR_WARPS * 32) dr_smem[i] = 0.f;
    pdl_wait();
    pdl_trigger();
    const int t0 = cu_seqlens[seq], t1 = cu_seqlens[seq + 1], slot = state_slots[seq];
    const bool wide = ((D | C | Dv) & 3) == 0 && !(((uintptr_t)y) & 15);
    float* st = state + (((size_t)slot * H + h) * Dv + (col < Dv ? col : 0)) * D;
    float S[R];
#pragma unroll
    for (int r = 0; r < R; ++r) S[r] = 0.f;
    if (col < Dv) {
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
            const int d = 4 * li + 32 * j;
            if ((D & 3) == 0) {
                if (d < D) {
                    const float4 s4 = *reinterpret_cast<const float4*>(st + d);
                    S[4 * j] = s4.x; S[4 * j + 1] = s4.y; S[4 * j + 2] = s4.z; S[4 * j + 3] = s4.w;
                }
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (d + e < D) S[4 * j + e] = st[d + e];
            }
        }
    }
    __syncthreads();   // (the zeros are there before the first copies)

    auto stage = [&](int buf, int tb) {
        const int n = min(DR_CHUNK, t1 - tb);
        float *qd = q_s + buf * DR_CHUNK * DP, *kd = k_s + buf * DR_CHUNK * DP, *vd = v_s + buf * DR_CHUNK * DR_COLS;
        const int vn = min(DR_COLS, Dv - col0);
        if (wide) {
            const int d4 = D >> 2, v4 = vn >> 2;
            for (int i = threadIdx.x; i < n * d4; i += DR_WARPS * 32) {
                const int tt = i / d4, d = (i - tt * d4) * 4;
                const float* src = y + (size_t)(tb + tt) * C + kvh * D + d;
                cp_async16(qd + tt * DP + d, src);
                cp_async16(kd + tt * DP + d, src + G * D);
            }
            for (int i = threadIdx.x; i < n * v4; i += DR_WARPS * 32) {
                const int tt = i / v4, c = (i - tt * v4) * 4;
                cp_async16(vd + tt * DR_COLS + c, y + (size_t)(tb + tt) * C + 2 * G * D + h * Dv + col0 + c);
            }
        } else {
            for (int i = threadIdx.x; i < n * D; i += DR_WARPS * 32) {
                const int tt = i / D, d = i - tt * D;
                const float* src = y + (size_t)(tb + tt) * C + kvh * D + d;
                dr_copy4(qd + tt * DP + d, src);
                dr_copy4(kd + tt * DP + d, src + G * D);
            }
            for (int i = threadIdx.x; i < n * vn; i += DR_WARPS * 32) {
                const int tt = i / vn, c = i - tt * vn;
                dr_copy4(vd + tt * DR_COLS + c, y + (size_t)(tb + tt) * C + 2 * G * D + h * Dv + col0 + c);
            }
        }
        for (int i = threadIdx.x; i < (DR_CHUNK - n) * DP; i += DR_WARPS * 32) {
            qd[n * DP + i] = 0.f;
            kd[n * DP + i] = 0.f;
        }
        for (int i = threadIdx.x; i < (DR_CHUNK - n) * DR_COLS; i += DR_WARPS * 32) vd[n * DR_COLS + i] = 0.f;
        cp_async_commit();
    };
    auto ask = [&](DrGates& g, int tb) {   // lane tt: token tb + tt
        const int t = tb + lane;
        if (lane < DR_CHUNK && t < t1) {
            g.a = ab[(size_t)t * ldab + a_col + h];
            g.b = ab[(size_t)t * ldab + b_col + h];
            const float* d = dots + ((size_t)t * G + kvh) * DR_DOTS;
#pragma unroll
            for (int i = 0; i < 3; ++i) g.kk[i] = d[i];
#pragma unroll
            for (int i = 0; i < 4; ++i) g.qk[i] = d[3 + i];
        }
    };
    auto coefficients = [&](const DrGates& g, int buf, int tb) {
        const bool there = lane < DR_CHUNK && tb + lane < t1;
        const float gt = there ? expf(neg_a * dr_softplus(g.a + bias)) : 1.f;
        const float beta = there ? 1.f / (1.f + expf(-g.b)) : 0.f;
        const int i = lane & 3;
        float gs[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) gs[j] = __shfl_sync(0xffffffffu, gt, (lane & ~3) + j);
        float gamma = 1.f, after = 1.f, rho[4] = {1.f, 1.f, 1.f, 1.f};   // rho[j]: decays after j up to i
#pragma unroll
        for (int l = 0; l < 4; ++l) {
            if (l <= i) gamma *= gs[l]; else after *= gs[l];
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (l > j && l <= i) rho[j] *= gs[l];
        }
        float bk[3], qk[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            // the product with token j of the mini-chunk, i - j tokens back
            float kd = 0.f, qd = 0.f;
#pragma unroll
            for (int b = 0; b < 4; ++b)
                if (i - j == b) { qd = g.qk[b]; if (b) kd = g.kk[b > 0 ? b - 1 : 0]; }
            if (j < 3) bk[j] = there && j < i ? beta * rho[j] * kd : 0.f;
            qk[j] = there && j <= i ? rho[j] * qd : 0.f;
        }
        if (lane < DR_CHUNK) {
            float4* dst = reinterpret_cast<float4*>(c_s + (buf * DR_CHUNK + lane) * DR_COEF);
            dst[0] = make_float4(beta * gamma, beta, after, gamma);
            dst[1] = make_float4(bk[0], bk[1], bk[2], 0.f);
            dst[2] = make_float4(qk[0], qk[1], qk[2], qk[3]);
        }
    };

    if (t1 > t0) {
        stage(0, t0);
        if (warp == 0) {
            DrGates g = {};
            ask(g, t0);
            coefficients(g, 0, t0);
        }
    }
    int buf = 0, turn = 1;
    for (int tb = t0; tb < t1; tb += DR_CHUNK, buf ^= 1, turn = (turn + 1) & (DR_WARPS - 1)) {
        const int n = min(DR_CHUNK, t1 - tb);
        const bool more = tb + DR_CHUNK < t1;
        cp_async_wait<0>();
        __syncthreads();
        DrGates g = {};
        if (more) {
            stage(buf ^ 1, tb + DR_CHUNK);
            if (warp == turn) ask(g, tb + DR_CHUNK);
        }
        const float *qb = q_s + buf * DR_CHUNK * DP + 4 * li, *kb = k_s + buf * DR_CHUNK * DP + 4 * li;
        const float *vb = v_s + buf * DR_CHUNK * DR_COLS + cl, *cb = c_s + buf * DR_CHUNK * DR_COEF;
        for (int m = 0; m < n; m += DR_MINI) {
            constexpr bool KEEP = R <= 16;   // the keys stay in registers from the products to the update
            float kreg[KEEP ? DR_MINI : 1][KEEP ? R : 1];
            float p[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) p[i] = 0.f;
#pragma unroll
            for (int j = 0; j < R / 4; ++j) {
#pragma unroll
                for (int i = 0; i < DR_MINI; ++i) {
                    const float4 k4 = *reinterpret_cast<const float4*>(kb + (m + i) * DP + 32 * j);
                    const float4 q4 = *reinterpret_cast<const float4*>(qb + (m + i) * DP + 32 * j);
                    if (KEEP) {
                        kreg[KEEP ? i : 0][KEEP ? 4 * j : 0] = k4.x;
                        kreg[KEEP ? i : 0][KEEP ? 4 * j + 1 : 0] = k4.y;
                        kreg[KEEP ? i : 0][KEEP ? 4 * j + 2 : 0] = k4.z;
                        kreg[KEEP ? i : 0][KEEP ? 4 * j + 3 : 0] = k4.w;
                    }
                    p[i] = fmaf(S[4 * j], k4.x, p[i]); p[i] = fmaf(S[4 * j + 1], k4.y, p[i]);
                    p[i] = fmaf(S[4 * j + 2], k4.z, p[i]); p[i] = fmaf(S[4 * j + 3], k4.w, p[i]);
                    p[4 + i] = fmaf(S[4 * j], q4.x, p[4 + i]); p[4 + i] = fmaf(S[4 * j + 1], q4.y, p[4 + i]);
                    p[4 + i] = fmaf(S[4 * j + 2], q4.z, p[4 + i]); p[4 + i] = fmaf(S[4 * j + 3], q4.w, p[4 + i]);
                }
            }
            // the eight sums over the column's eight lanes: lane i ends with the sum number i
            float a4[4], a2[2], mine;
            const bool h4 = lane & 4, h2 = lane & 2, h1 = lane & 1;
#pragma unroll
            for (int i = 0; i < 4; ++i) a4[i] = (h4 ? p[4 + i] : p[i]) + __shfl_xor_sync(0xffffffffu, h4 ? p[i] : p[4 + i], 4);
#pragma unroll
            for (int i = 0; i < 2; ++i) a2[i] = (h2 ? a4[2 + i] : a4[i]) + __shfl_xor_sync(0xffffffffu, h2 ? a4[i] : a4[2 + i], 2);
            mine = (h1 ? a2[1] : a2[0]) + __shfl_xor_sync(0xffffffffu, h1 ? a2[0] : a2[1], 1);
            float u[4], wu[4], gamma_all = 1.f;
#pragma unroll
            for (int i = 0; i < DR_MINI; ++i) {
                const float4 c0 = *reinterpret_cast<const float4*>(cb + (m + i) * DR_COEF);
                const float kS = __shfl_sync(0xffffffffu, mine, i, 8);
                float v = fmaf(-c0.x, kS, c0.y * vb[(m + i) * DR_COLS]);
                if (i > 0) {
                    const float4 c1 = *reinterpret_cast<const float4*>(cb + (m + i) * DR_COEF + 4);
                    v = fmaf(-c1.x, u[0], v);
                    if (i > 1) v = fmaf(-c1.y, u[1], v);
                    if (i > 2) v = fmaf(-c1.z, u[2], v);
                }
                u[i] = v;
                wu[i] = c0.z * v;
                if (i == DR_MINI - 1) gamma_all = c0.w;
            }
            if (li >= 4) {
                const int tt = m + li - 4;
                const float gamma = cb[tt * DR_COEF + 3];
                const float4 c2 = *reinterpret_cast<const float4*>(cb + tt * DR_COEF + 8);
                float o = gamma * mine;
                o = fmaf(c2.x, u[0], o); o = fmaf(c2.y, u[1], o); o = fmaf(c2.z, u[2], o); o = fmaf(c2.w, u[3], o);
                if (tt < n && col < Dv) out[((size_t)(tb + tt) * H + h) * Dv + col] = o;
            }
#pragma unroll
            for (int j = 0; j < R / 4; ++j) {
#pragma unroll
                for (int e = 0; e < 4; ++e) S[4 * j + e] *= gamma_all;
#pragma unroll
                for (int i = 0; i < DR_MINI; ++i) {
                    float kk[4];
                    if (KEEP) {
#pragma unroll
                        for (int e = 0; e < 4; ++e) kk[e] = kreg[KEEP ? i : 0][KEEP ? 4 * j + e : 0];
                    } else {
                        const float4 k4 = *reinterpret_cast<const float4*>(kb + (m + i) * DP + 32 * j);
                        kk[0] = k4.x; kk[1] = k4.y; kk[2] = k4.z; kk[3] = k4.w;
                    }
#pragma unroll
                    for (int e = 0; e < 4; ++e) S[4 * j + e] = fmaf(kk[e], wu[i], S[4 * j + e]);
                }
            }
        }
        if (more && warp == turn) coefficients(g, buf ^ 1, tb + DR_CHUNK);
    }
    if (col < Dv) {
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
            const int d = 4 * li + 32 * j;
            if ((D & 3) == 0) {
                if (d < D) *reinterpret_cast<float4*>(st + d) = make_float4(S[4 * j], S[4 * j + 1], S[4 * j + 2], S[4 * j + 3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (d + e < D) st[d + e] = S[4 * j + e];
            }
        }
    }
    // the request's last inputs of the convolutions, its blocks sharing the channels
    const int part = blockIdx.y * gridDim.x + blockIdx.x, parts = gridDim.x * gridDim.y;
    for (int c = part * DR_WARPS * 32 + threadIdx.x; c < C; c += parts * DR_WARPS * 32)
        for (int t = max(t0, t1 - (taps - 1)); t < t1; ++t)
            ring[((size_t)slot * taps + positions[t] % taps) * C + c] =
                x_bf16 ? to_f32(((const bf16*)x)[(size_t)t * ldx + c]) : ((const float*)x)[(size_t)t * ldx + c];
}

// neg_exp_a, dt_bias float32 [H]: -exp(A_log) and the decay's offset.  ab float32 [tokens, ldab]: a and b of head h in columns
// a_col + h, b_col + h.  y, dots: from `vx_delta_conv` of the same step; x, ldx: what that read.  state float32
// [slots, H, Dv, D], ring float32 [slots, taps, C]: read and written.  out float32 [tokens, H * Dv].
extern "C" int vx_delta_walk(const float* y, const float* dots, const float* ab, int ldab, int a_col, int b_col,
                             const float* neg_exp_a, const float* dt_bias, float* state, float* ring, const void* x, int ldx,
                             const int* cu_seqlens, const int* state_slots, const int* positions, float* out, int seqs, int G, int D,
                             int H, int Dv, int taps, int dtype, cudaStream_t stream) {
    if (seqs <= 0) return VX_OK;
    if (G <= 0 || D <= 0 || H <= 0 || Dv <= 0 || H % G || taps <= 0) return VX_ERR_SHAPE;
    if (ldab < a_col + H || ldab < b_col + H || a_col < 0 || b_col < 0 || ldx < 2 * G * D + H * Dv) return VX_ERR_SHAPE;
    if (D > 256 || taps > DR_MAX_TAPS || seqs > 65535 || H > 65535) return VX_ERR_LIMIT;
    if (dtype != VX_F32 && dtype != VX_BF16) return VX_ERR_DTYPE;
    static bool configured[4][VX_MAX_DEVICES];
    dim3 grid((Dv + DR_COLS - 1) / DR_COLS, H, seqs);
#define DR_GO(R_, SLOT)                                                                                                       \
    do {                                                                                                                      \
        if (int rc = vx_configure_smem(delta_walk_kernel<R_>, DR_SMEM(8 * R_), configured[SLOT])) return rc;                  \
        VX_LAUNCH_K(VX_K_ATTENTION, (delta_walk_kernel<R_>), grid, DR_WARPS * 32, DR_SMEM(8 * R_), stream, y, dots, ab, ldab, \
                    a_col, b_col, neg_exp_a, dt_bias, state, ring, x, ldx, dtype == VX_BF16 ? 1 : 0, cu_seqlens, state_slots, \
                    positions, out, G, D, H, Dv, taps);                                                                       \
    } while (0)
    if (D <= 32) DR_GO(4, 3);
    else if (D <= 64) DR_GO(8, 0);
    else if (D <= 128) DR_GO(16, 1);
    else DR_GO(32, 2);
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
