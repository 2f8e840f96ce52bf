// Token shift: what a sublayer reads is moved towards the token before it, channel by channel.
//
//   n_t  = RMS norm of the stream's row t, times w
//   h_t  = n_t + (n_(t-1) - n_t) * mu                        (n_(-1) = 0)
//   m_it = h_t + (h_(t-1) - h_t) * nu_i,  i = 0 .. mixes - 1   (h_(-1) = 0; for a mixer that shifts its input again, with a
//                                                              vector of its own for every projection)
//
// shift_norm      residual update (residual + delta), norm, shift and, with `mixes`, the second shift's m_i, in one pass
// shift_mix       the second shift alone, on rows that are already normed
// shift_commit    the last rows' n and h into the requests' slots, for requests that several blocks worked on
// low_rank_decay  -exp(tanh(a) W + b): the logarithm of a decay per channel, from a projection through a narrow middle
//
// A request's last n (and h) lie in float32 in its state slot.  shift_norm: a block takes R consecutive rows of the step,
// a thread the same channels of each, so the row before is in registers; the rows just before the block's first are
// normed again by this block (the stream is read from `res_in` and written to `res_out`, so no block sees another's
// update).  A request whose rows of this step lie in one block has its slot written there; the others' last rows go to
// `save` and from there into the slots by shift_commit, after every block has read its slots.
// A row's norm is the same bits whichever block computes it, so results do not depend on how a request was cut.
#include "common.cuh"

#define TS_MAX_THREADS 512
#define TS_MAX_GROUPS 8      // groups of V channels a thread owns at most
#define TS_MAX_MIXES 8

template <int V> __device__ __forceinline__ void ts_load(const float* p, float (&v)[V]) {
    if constexpr (V == 4) { const float4 t = *reinterpret_cast<const float4*>(p); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w; }
    else v[0] = p[0];
}
template <int V> __device__ __forceinline__ void ts_load(const bf16* p, float (&v)[V]) {
    if constexpr (V == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
    } else v[0] = __bfloat162float(p[0]);
}
template <int V> __device__ __forceinline__ void ts_store(float* p, const float (&v)[V]) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else p[0] = v[0];
}
template <int V> __device__ __forceinline__ void ts_store(bf16* p, const float (&v)[V]) {
    if constexpr (V == 4) {
        uint2 raw;
        *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v[0], v[1]);
        *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = raw;
    } else p[0] = __float2bfloat16_rn(v[0]);
}

struct TsStep {
    const int* seq_of_token;
    const int* cu_seqlens;
    const int* state_slots;
    int tokens;
};

// a + (b - a) * m
__device__ __forceinline__ float ts_mix(float a, float b, float m) { return fmaf(b - a, m, a); }

// (blocks an SM: rows of one group a thread without mixes leave registers for three)
template <typename T, int V, int NG, bool MIX>
__global__ void __launch_bounds__(TS_MAX_THREADS, NG == 1 ? (MIX ? 2 : 3) : 1)
shift_norm_kernel(const float* __restrict__ res_in, const T* __restrict__ delta, float* __restrict__ res_out,
                  const float* __restrict__ w, float eps, const float* __restrict__ mu, const float* __restrict__ nu, int mixes,
                  TsStep st, float* state_n, float* state_h, float* __restrict__ save, T* __restrict__ out, int E, int R) {
    __shared__ float scratch[2][TS_MAX_THREADS / 32];
    const int t0 = blockIdx.x * R, t1 = min(st.tokens, t0 + R);
    int at[NG];
    bool in[NG];
    float g[NG][V], m[NG][V];
#pragma unroll
    for (int j = 0; j < NG; ++j) {
        at[j] = (threadIdx.x + j * blockDim.x) * V;
        in[j] = at[j] < E;
#pragma unroll
        for (int e = 0; e < V; ++e) { g[j][e] = 0.f; m[j][e] = 0.f; }
        if (in[j]) { ts_load<V>(w + at[j], g[j]); ts_load<V>(mu + at[j], m[j]); }
    }
    pdl_wait();
    pdl_trigger();
    // the stream's row t after this step's update, as it is read (no sum yet)
    auto fetch = [&](int t, float (&v)[NG][V]) {
#pragma unroll
        for (int j = 0; j < NG; ++j) {
#pragma unroll
            for (int e = 0; e < V; ++e) v[j][e] = 0.f;
            if (!in[j]) continue;
            ts_load<V>(res_in + (size_t)t * E + at[j], v[j]);
            if (delta) {
                float d[V];
                ts_load<V>(delta + (size_t)t * E + at[j], d);
#pragma unroll
                for (int e = 0; e < V; ++e) v[j][e] += d[e];
            }
        }
    };
    // One barrier a row: the warps' sums of consecutive rows go to two buffers in turn (when a buffer is written again, every
    // thread has passed the barrier after its last reading).
    int turn = 0;
    const int warps = blockDim.x >> 5, lane = threadIdx.x & 31;
    auto norm = [&](float (&v)[NG][V]) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < NG; ++j)
#pragma unroll
            for (int e = 0; e < V; ++e) ss = fmaf(v[j][e], v[j][e], ss);
        ss = warp_sum(ss);
        if (lane == 0) scratch[turn][threadIdx.x >> 5] = ss;
        __syncthreads();
        ss = warp_sum(lane < warps ? scratch[turn][lane] : 0.f);
        turn ^= 1;
        const float rstd = rsqrtf(ss / (float)E + eps);
#pragma unroll
        for (int j = 0; j < NG; ++j)
#pragma unroll
            for (int e = 0; e < V; ++e) v[j][e] = v[j][e] * rstd * g[j][e];
    };
    auto from_slot = [&](const float* state, int slot, float (&v)[NG][V]) {
#pragma unroll
        for (int j = 0; j < NG; ++j)
            if (in[j]) ts_load<V>(state + (size_t)slot * E + at[j], v[j]);
    };
    int seq = st.seq_of_token[t0], first = st.cu_seqlens[seq], end = st.cu_seqlens[seq + 1], slot = st.state_slots[seq];
    float np[NG][V], hp[NG][V], cur[NG][V], nxt[NG][V];   // the row before: normed, shifted
#pragma unroll
    for (int j = 0; j < NG; ++j)
#pragma unroll
        for (int e = 0; e < V; ++e) { np[j][e] = 0.f; hp[j][e] = 0.f; }
    fetch(t0, cur);
    if (t0 == first) {
        from_slot(state_n, slot, np);
        if (MIX) from_slot(state_h, slot, hp);
    } else {
        fetch(t0 - 1, np);
        if (MIX) {
            if (t0 - 1 == first) from_slot(state_n, slot, hp);
            else { fetch(t0 - 2, hp); norm(hp); }
        }
        norm(np);
        if (MIX) {
#pragma unroll
            for (int j = 0; j < NG; ++j)
#pragma unroll
                for (int e = 0; e < V; ++e) hp[j][e] = ts_mix(np[j][e], hp[j][e], m[j][e]);
        }
    }
    for (int t = t0; t < t1; ++t) {
        if (t == end) {   // the next request of the step begins inside this block
            seq = st.seq_of_token[t];
            first = t;
            end = st.cu_seqlens[seq + 1];
            slot = st.state_slots[seq];
            from_slot(state_n, slot, np);
            if (MIX) from_slot(state_h, slot, hp);
        }
        if (t + 1 < t1) fetch(t + 1, nxt);
        if (delta) {
#pragma unroll
            for (int j = 0; j < NG; ++j)
                if (in[j]) ts_store<V>(res_out + (size_t)t * E + at[j], cur[j]);
        }
        norm(cur);
#pragma unroll
        for (int j = 0; j < NG; ++j) {
            float h[V];
#pragma unroll
            for (int e = 0; e < V; ++e) h[e] = ts_mix(cur[j][e], np[j][e], m[j][e]);
            if (in[j]) {
                if (!MIX) {
                    ts_store<V>(out + (size_t)t * E + at[j], h);
                } else {
                    for (int i = 0; i < mixes; ++i) {
                        float c[V], y[V];
                        ts_load<V>(nu + (size_t)i * E + at[j], c);
#pragma unroll
                        for (int e = 0; e < V; ++e) y[e] = ts_mix(h[e], hp[j][e], c[e]);
                        ts_store<V>(out + ((size_t)i * st.tokens + t) * E + at[j], y);
                    }
                }
            }
#pragma unroll
            for (int e = 0; e < V; ++e) { np[j][e] = cur[j][e]; hp[j][e] = h[e]; cur[j][e] = nxt[j][e]; }
        }
        if (t + 1 == end) {
            const bool mine = first >= t0;   // all of the request's rows are this block's
            float* dn = mine ? state_n + (size_t)slot * E : save + (size_t)seq * 2 * E;
            float* dh = mine ? (state_h ? state_h + (size_t)slot * E : nullptr) : save + ((size_t)seq * 2 + 1) * E;
#pragma unroll
            for (int j = 0; j < NG; ++j) {
                if (!in[j]) continue;
                ts_store<V>(dn + at[j], np[j]);
                if (MIX) ts_store<V>(dh + at[j], hp[j]);
            }
        }
    }
}

// One block per request: the rows that shift_norm left in `save` for requests whose rows lie in more than one block of R.
__global__ void shift_commit_kernel(const float* __restrict__ save, const int* __restrict__ cu_seqlens,
                                    const int* __restrict__ state_slots, float* __restrict__ state_n, float* __restrict__ state_h,
                                    int E, int R) {
    pdl_wait();
    pdl_trigger();
    const int s = blockIdx.x, a = cu_seqlens[s], b = cu_seqlens[s + 1];
    if (b <= a || a / R == (b - 1) / R) return;
    const size_t slot = state_slots[s];
    for (int i = threadIdx.x; i < E; i += blockDim.x) {
        state_n[slot * E + i] = save[(size_t)s * 2 * E + i];
        if (state_h) state_h[slot * E + i] = save[((size_t)s * 2 + 1) * E + i];
    }
}

// rows of a block of shift_norm: enough blocks to fill the SMs a few times over, at most 8 rows
static int ts_rows_per_block(int tokens, int sms) {
    const int r = tokens / (4 * sms);
    return r < 1 ? 1 : (r > 8 ? 8 : r);
}

template <typename T>
static int launch_shift_norm(const float* res_in, const T* delta, float* res_out, const float* w, float eps, const float* mu,
                             const float* nu, int mixes, TsStep st, int seqs, int max_new, float* state_n, float* state_h,
                             float* save, T* out, int E, cudaStream_t stream) {
    static int sms[VX_MAX_DEVICES];
    const int R = max_new == 1 ? 1 : ts_rows_per_block(st.tokens, vx_sm_count(sms));
    const uintptr_t all = (uintptr_t)res_in | (uintptr_t)res_out | (uintptr_t)w | (uintptr_t)mu | (uintptr_t)nu | (uintptr_t)state_n |
                          (uintptr_t)state_h | (uintptr_t)save;
    const bool vec = E % 4 == 0 && !(all & 15) && !(((uintptr_t)delta | (uintptr_t)out) & (4 * sizeof(T) - 1));
    const int groups = vec ? E / 4 : E;
    int ng = 1;
    while (ng < TS_MAX_GROUPS && groups > ng * TS_MAX_THREADS) ng *= 2;
    if (groups > ng * TS_MAX_THREADS) return VX_ERR_LIMIT;
    int threads = ((groups + ng - 1) / ng + 31) / 32 * 32;
    const int blocks = (st.tokens + R - 1) / R;
#define TS_GO(V_, NG_)                                                                                                         \
    do {                                                                                                                       \
        if (mixes)                                                                                                             \
            VX_LAUNCH_K(VX_K_ELEMENTWISE, (shift_norm_kernel<T, V_, NG_, true>), blocks, threads, 0, stream, res_in, delta,    \
                        res_out, w, eps, mu, nu, mixes, st, state_n, state_h, save, out, E, R);                                \
        else                                                                                                                   \
            VX_LAUNCH_K(VX_K_ELEMENTWISE, (shift_norm_kernel<T, V_, NG_, false>), blocks, threads, 0, stream, res_in, delta,   \
                        res_out, w, eps, mu, nu, mixes, st, state_n, state_h, save, out, E, R);                                \
    } while (0)
#define TS_GO_V(V_)                                                                                                            \
    do {                                                                                                                       \
        if (ng == 1) TS_GO(V_, 1); else if (ng == 2) TS_GO(V_, 2); else if (ng == 4) TS_GO(V_, 4); else TS_GO(V_, 8);          \
    } while (0)
    if (vec) TS_GO_V(4); else TS_GO_V(1);
#undef TS_GO_V
#undef TS_GO
    if (max_new > 1 && st.tokens > R)   // (a request may lie in several blocks)
        VX_LAUNCH_K(VX_K_ELEMENTWISE, shift_commit_kernel, seqs, 256, 0, stream, (const float*)save, st.cu_seqlens, st.state_slots,
                    state_n, mixes ? state_h : (float*)nullptr, E, R);
    VX_LAUNCH_CHECK();
    return VX_OK;
}

// res_in float32 [tokens, E]; with delta (T) the sum goes to res_out (another buffer), without one nothing is written there.
// out T [tokens, E], or with mixes > 0 (nu float32 [mixes, E], state_h) [mixes, tokens, E].  state_n, state_h float32
// [slots, E]; save float32 [seqs, 2, E], needed for max_new > 1.
extern "C" int vx_shift_norm(const float* res_in, const void* delta, float* res_out, const float* w, float eps, const float* mu,
                             const float* nu, int mixes, const int* seq_of_token, const int* cu_seqlens, const int* state_slots,
                             int seqs, int max_new, float* state_n, float* state_h, float* save, void* out, int tokens, int E,
                             int dtype, cudaStream_t stream) {
    if (tokens <= 0 || seqs <= 0) return VX_OK;
    if (E <= 0 || mixes < 0 || mixes > TS_MAX_MIXES || max_new <= 0 || !mu || !state_n || (mixes && (!nu || !state_h))) return VX_ERR_SHAPE;
    if (delta && (!res_out || res_out == res_in)) return VX_ERR_SHAPE;
    if (max_new > 1 && !save) return VX_ERR_SHAPE;
    TsStep st = {seq_of_token, cu_seqlens, state_slots, tokens};
    if (dtype == VX_F32)
        return launch_shift_norm<float>(res_in, (const float*)delta, res_out, w, eps, mu, nu, mixes, st, seqs, max_new, state_n,
                                        state_h, save, (float*)out, E, stream);
    if (dtype == VX_BF16)
        return launch_shift_norm<bf16>(res_in, (const bf16*)delta, res_out, w, eps, mu, nu, mixes, st, seqs, max_new, state_n,
                                       state_h, save, (bf16*)out, E, stream);
    return VX_ERR_DTYPE;
}

// One block per row: out[i, t] = x_t + (x_(t-1) - x_t) * nu_i, the row before a request's first being its slot's.
template <typename T>
__global__ void shift_mix_kernel(const T* __restrict__ x, const float* __restrict__ nu, int mixes, TsStep st,
                                 const float* __restrict__ state_h, T* __restrict__ out, int E) {
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x, seq = st.seq_of_token[t];
    const bool opens = t == st.cu_seqlens[seq];
    const float* prev = state_h + (size_t)st.state_slots[seq] * E;
    for (int c = threadIdx.x; c < E; c += blockDim.x) {
        const float a = to_f32(x[(size_t)t * E + c]);
        const float b = opens ? prev[c] : to_f32(x[(size_t)(t - 1) * E + c]);
        for (int i = 0; i < mixes; ++i) out[((size_t)i * st.tokens + t) * E + c] = from_f32<T>(ts_mix(a, b, nu[(size_t)i * E + c]));
    }
}
template <typename T>
__global__ void shift_keep_kernel(const T* __restrict__ x, const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots,
                                  float* __restrict__ state_h, int E) {
    pdl_wait();
    pdl_trigger();
    const int s = blockIdx.x, last = cu_seqlens[s + 1] - 1;
    if (last < cu_seqlens[s]) return;
    for (int c = threadIdx.x; c < E; c += blockDim.x) state_h[(size_t)state_slots[s] * E + c] = to_f32(x[(size_t)last * E + c]);
}

extern "C" int vx_shift_mix(const void* x, const float* nu, int mixes, const int* seq_of_token, const int* cu_seqlens,
                            const int* state_slots, int seqs, float* state_h, void* out, int tokens, int E, int dtype,
                            cudaStream_t stream) {
    if (tokens <= 0 || seqs <= 0) return VX_OK;
    if (E <= 0 || mixes <= 0 || mixes > TS_MAX_MIXES || !nu || !state_h) return VX_ERR_SHAPE;
    TsStep st = {seq_of_token, cu_seqlens, state_slots, tokens};
    const int threads = E >= 1024 ? 256 : 128;
    if (dtype == VX_F32) {
        VX_LAUNCH_K(VX_K_ELEMENTWISE, (shift_mix_kernel<float>), tokens, threads, 0, stream, (const float*)x, nu, mixes, st,
                    (const float*)state_h, (float*)out, E);
        VX_LAUNCH_K(VX_K_ELEMENTWISE, (shift_keep_kernel<float>), seqs, threads, 0, stream, (const float*)x, cu_seqlens, state_slots, state_h, E);
    } else if (dtype == VX_BF16) {
        VX_LAUNCH_K(VX_K_ELEMENTWISE, (shift_mix_kernel<bf16>), tokens, threads, 0, stream, (const bf16*)x, nu, mixes, st,
                    (const float*)state_h, (bf16*)out, E);
        VX_LAUNCH_K(VX_K_ELEMENTWISE, (shift_keep_kernel<bf16>), seqs, threads, 0, stream, (const bf16*)x, cu_seqlens, state_slots, state_h, E);
    } else {
        return VX_ERR_DTYPE;
    }
    VX_LAUNCH_CHECK();
    return VX_OK;
}

// log a[t, c] = -exp(b[c] + sum_r tanh(x[t, r]) w[r, c]), all float32.  A block takes TOK tokens by LD_THREADS * CH
// channels: the tokens' tanh in shared memory, the sums of CH channels a thread in registers, w read once per block
// (coalesced: it is stored [rank, channels]).  r runs upwards, so a token's result does not depend on the tokens beside it.
#define LD_THREADS 128
#define LD_AHEAD 4
template <int TOK, int CH>
__global__ void __launch_bounds__(LD_THREADS)
low_rank_decay_kernel(const float* __restrict__ x, int ldx, int rank, const float* __restrict__ w, const float* __restrict__ b,
                      float* __restrict__ out, int tokens, int C) {
    extern __shared__ __align__(16) float ld_s[];   // [rank][TOK]
    const int c0 = blockIdx.x * LD_THREADS * CH + threadIdx.x, t0 = blockIdx.y * TOK;
    float wv[LD_AHEAD][CH], acc[TOK][CH];
    bool in[CH];
#pragma unroll
    for (int j = 0; j < CH; ++j) {
        const int c = c0 + j * LD_THREADS;
        in[j] = c < C;
        const float b0 = in[j] ? b[c] : 0.f;
#pragma unroll
        for (int i = 0; i < TOK; ++i) acc[i][j] = b0;
#pragma unroll
        for (int u = 0; u < LD_AHEAD; ++u) wv[u][j] = (in[j] && u < rank) ? w[(size_t)u * C + c] : 0.f;   // (weights depend on no earlier kernel)
    }
    pdl_wait();
    pdl_trigger();
    for (int i = threadIdx.x; i < rank * TOK; i += LD_THREADS) {
        const int tt = i / rank, r = i - tt * rank;
        ld_s[r * TOK + tt] = t0 + tt < tokens ? tanhf(x[(size_t)(t0 + tt) * ldx + r]) : 0.f;
    }
    __syncthreads();
    for (int r0 = 0; r0 < rank; r0 += LD_AHEAD) {
        float nw[LD_AHEAD][CH];
#pragma unroll
        for (int u = 0; u < LD_AHEAD; ++u)
#pragma unroll
            for (int j = 0; j < CH; ++j)
                nw[u][j] = (in[j] && r0 + LD_AHEAD + u < rank) ? w[(size_t)(r0 + LD_AHEAD + u) * C + c0 + j * LD_THREADS] : 0.f;
#pragma unroll
        for (int u = 0; u < LD_AHEAD; ++u) {
            if (r0 + u < rank) {
                float th[TOK];
                if constexpr (TOK % 4 == 0) {
#pragma unroll
                    for (int i = 0; i < TOK; i += 4) {
                        const float4 t4 = *reinterpret_cast<const float4*>(ld_s + (r0 + u) * TOK + i);
                        th[i] = t4.x; th[i + 1] = t4.y; th[i + 2] = t4.z; th[i + 3] = t4.w;
                    }
                } else {
#pragma unroll
                    for (int i = 0; i < TOK; ++i) th[i] = ld_s[(r0 + u) * TOK + i];
                }
#pragma unroll
                for (int i = 0; i < TOK; ++i)
#pragma unroll
                    for (int j = 0; j < CH; ++j) acc[i][j] = fmaf(th[i], wv[u][j], acc[i][j]);
            }
        }
#pragma unroll
        for (int u = 0; u < LD_AHEAD; ++u)
#pragma unroll
            for (int j = 0; j < CH; ++j) wv[u][j] = nw[u][j];
    }
#pragma unroll
    for (int i = 0; i < TOK; ++i)
#pragma unroll
        for (int j = 0; j < CH; ++j)
            if (in[j] && t0 + i < tokens) out[(size_t)(t0 + i) * C + c0 + j * LD_THREADS] = -expf(acc[i][j]);
}

#define LD_MAX_RANK 1024
#define LD_FEW_TOKENS 16   // steps of up to so many tokens take small tiles
// x float32 [tokens, ldx] (the first `rank` columns), w float32 [rank, C], b float32 [C], out float32 [tokens, C].
extern "C" int vx_low_rank_decay(const float* x, int ldx, int rank, const float* w, const float* b, float* out, int tokens, int C,
                                 cudaStream_t stream) {
    if (tokens <= 0) return VX_OK;
    if (rank <= 0 || C <= 0 || ldx < rank) return VX_ERR_SHAPE;
    if (rank > LD_MAX_RANK || (tokens + 15) / 16 > 65535) return VX_ERR_LIMIT;
    static bool conf[2][VX_MAX_DEVICES];
    if (tokens <= LD_FEW_TOKENS) {
        if (int rc = vx_configure_smem(low_rank_decay_kernel<2, 1>, LD_MAX_RANK * 2 * sizeof(float), conf[0])) return rc;
        VX_LAUNCH_K(VX_K_ELEMENTWISE, (low_rank_decay_kernel<2, 1>), dim3((C + LD_THREADS - 1) / LD_THREADS, (tokens + 1) / 2), LD_THREADS,
                    (size_t)rank * 2 * sizeof(float), stream, x, ldx, rank, w, b, out, tokens, C);
    } else {
        if (int rc = vx_configure_smem(low_rank_decay_kernel<16, 2>, LD_MAX_RANK * 16 * sizeof(float), conf[1])) return rc;
        VX_LAUNCH_K(VX_K_ELEMENTWISE, (low_rank_decay_kernel<16, 2>), dim3((C + 2 * LD_THREADS - 1) / (2 * LD_THREADS), (tokens + 15) / 16),
                    LD_THREADS, (size_t)rank * 16 * sizeof(float), stream, x, ldx, rank, w, b, out, tokens, C);
    }
    VX_LAUNCH_CHECK();
    return VX_OK;
}
