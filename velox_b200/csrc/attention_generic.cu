// Paged causal attention, the general kernel: any head size up to 256 (values may
// have another size than keys), any number of heads and groups, any page size, an
// optional window with optionally kept first positions, an optional bias by distance,
// element type float or bfloat16.  It serves prompt portions and decoded
// tokens alike, and it is the whole of the 32-bit path.
//
// One block per (token, query head).  The token's absolute position p gives its
// keys: j in [start, p], start = max(0, p + 1 - window) with a window, else 0; with
// keep_first > 0 also j in [0, min(keep_first, start)), at their true positions.  With
// chunk > 0 start is no less than p - p mod chunk: a token sees its own run of `chunk`
// positions only, the runs counted from the request's position 0.
// Key j of the token's request lies in page block_table[seq, j / S] at offset
// j % S; pools are [page, Hk, S, D] and [page, Hk, S, Dv]; query head h reads kv head
// h / (H / Hk).  score = q.k * scale - slope_h * (p - j) with
// slope_h = 2^(-bias_exp * (h + 1) / H), or no bias for bias_exp = 0.
// With `sinks` (a float32 per query head) the softmax's denominator also holds
// exp(sinks[h]): an entry without a key or a value, not scaled.  With gate_col >= 0
// head h's output is multiplied by sigmoid(g), g the element at column gate_col + h
// of the token's row of `q`.  With softcap c > 0 a scaled score s becomes c tanh(s / c) before
// anything else is done to it.  A value row starts every v_stride elements (Dv unless the caller
// says otherwise: a pool whose rows hold the value as the first Dv elements of the key, v_pool =
// k_pool and v_stride = D, is read as it lies).
//
// Each warp takes chunks of 32 keys (chunk c goes to warp c mod 4), one key per
// lane: the lane forms the whole dot product q.k in float32, the warp keeps a
// running maximum m, sum l and accumulator acc (online softmax), and adds the
// 32 values in key order.  The four warps' (m, l, acc) are merged in warp
// order.  The order of every addition depends only on the token's own key
// range, never on the batch around it, so a position's output is bit-identical
// however the tokens were cut into steps.
#include "common.cuh"

#define ATT_WARPS 4
#define ATT_MAX_D 256

template <typename T>
__global__ void paged_attention_generic_kernel(
    const T* __restrict__ q, int q_row_stride, const T* __restrict__ k_pool,
    const T* __restrict__ v_pool, const int* __restrict__ block_table, int max_blocks,
    const int* __restrict__ seq_of_token, const int* __restrict__ positions, T* __restrict__ out,
    int out_row_stride, float scale, int window, int H, int Hk, int D, int S, int Dv, int keep_first,
    float bias_exp, const float* __restrict__ sinks, int gate_col, float softcap, int v_stride, int v_share, int out_f32,
    int chunk) {
    pdl_wait();
    pdl_trigger();
    __shared__ float q_s[ATT_MAX_D];
    __shared__ float acc_s[ATT_WARPS][ATT_MAX_D];
    __shared__ float m_s[ATT_WARPS], l_s[ATT_WARPS];

    const int t = blockIdx.x, h = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int hk = h / (H / Hk);
    const int seq = seq_of_token[t];
    const int kv_len = positions[t] + 1;
    int start = (window > 0 && kv_len > window) ? kv_len - window : 0;
    if (chunk > 0) start = max(start, kv_len - 1 - (kv_len - 1) % chunk);
    const int nkept = min(keep_first, start);   // kept first positions that lie before the window
    const float slope = bias_exp > 0.f ? exp2f(-bias_exp * (float)(h + 1) / (float)H) : 0.f;
    const int* bt = block_table + (size_t)seq * max_blocks;

    for (int d = threadIdx.x; d < D; d += blockDim.x)
        q_s[d] = to_f32(q[(size_t)t * q_row_stride + (size_t)h * D + d]);
    __syncthreads();

    constexpr int NR = ATT_MAX_D / 32;
    float acc[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) acc[i] = 0.f;
    float m = -INFINITY, l = 0.f;

    const int nkeys = nkept + kv_len - start;   // the n-th visible key is j = n (kept) or start + n - nkept
    const int nchunks = (nkeys + 31) >> 5;
    for (int c = warp; c < nchunks; c += ATT_WARPS) {
        const int n = c * 32 + lane;
        const int j = n < nkept ? n : start + n - nkept;
        const bool valid = n < nkeys;
        size_t base = 0;
        float s = -INFINITY;
        if (valid) {
            const int page = bt[j / S];
            base = ((size_t)page * Hk + hk) * S + (j % S);
            const T* kp = k_pool + base * D;
            if (v_share > 1) base = ((size_t)page * (Hk / v_share) + hk / v_share) * S + (j % S);
            float dot = 0.f;
            for (int d = 0; d < D; ++d) dot += q_s[d] * to_f32(kp[d]);
            s = dot * scale;
            if (softcap > 0.f) s = softcap * tanhf(s / softcap);
            s -= slope * (float)(kv_len - 1 - j);
        }
        const float m_new = fmaxf(m, warp_max(s));
        const float p = valid ? expf(s - m_new) : 0.f;
        const float alpha = expf(m - m_new);  // m = -inf on the first chunk: 0
        l = l * alpha + warp_sum(p);
#pragma unroll
        for (int i = 0; i < NR; ++i) acc[i] *= alpha;
        const int nvalid = min(32, nkeys - c * 32);
        for (int jj = 0; jj < nvalid; ++jj) {
            const float pj = __shfl_sync(0xffffffffu, p, jj);
            const size_t bj = __shfl_sync(0xffffffffu, (unsigned long long)base, jj);
            const T* vp = v_pool + bj * v_stride;
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                const int d = lane + 32 * i;
                if (d < Dv) acc[i] += pj * to_f32(vp[d]);
            }
        }
        m = m_new;
    }

    if (lane == 0) { m_s[warp] = m; l_s[warp] = l; }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = lane + 32 * i;
        if (d < Dv) acc_s[warp][d] = acc[i];
    }
    __syncthreads();
    float M = -INFINITY;
    for (int w = 0; w < ATT_WARPS; ++w) M = fmaxf(M, m_s[w]);
    float L = 0.f;
    float wgt[ATT_WARPS];
    for (int w = 0; w < ATT_WARPS; ++w) {
        wgt[w] = (m_s[w] == -INFINITY) ? 0.f : expf(m_s[w] - M);
        L += l_s[w] * wgt[w];
    }
    if (sinks) {
        // the sink joins the denominator only; where it exceeds every score the reference moves to it
        const float sk = sinks[h];
        if (sk > M) {
            const float f = expf(M - sk);   // (M is finite: a token always sees itself)
            L = L * f + 1.f;
            for (int w = 0; w < ATT_WARPS; ++w) wgt[w] *= f;
        } else {
            L += expf(sk - M);
        }
    }
    float gate = 1.f;
    if (gate_col >= 0) gate = 1.f / (1.f + expf(-to_f32(q[(size_t)t * q_row_stride + gate_col + h])));
    for (int d = threadIdx.x; d < Dv; d += blockDim.x) {
        float o = 0.f;
        for (int w = 0; w < ATT_WARPS; ++w) o += acc_s[w][d] * wgt[w];
        if (out_f32) reinterpret_cast<float*>(out)[(size_t)t * out_row_stride + (size_t)h * Dv + d] = o / L * gate;
        else out[(size_t)t * out_row_stride + (size_t)h * Dv + d] = from_f32<T>(o / L * gate);
    }
}

// `v_share` > 1: that many consecutive key heads read one value head (the value pool has Hk / v_share heads);
// `out_f32`: the output is written as float32 whatever the element type of the inputs; `chunk` > 0: see
// the top (it does not go with kept first positions).
extern "C" int vx_paged_attention_generic_chunk(const void* q, int q_row_stride, const void* k_pool,
                                                 const void* v_pool, const int* block_table, int max_blocks,
                                                 const int* seq_of_token, const int* positions, void* out,
                                                 int out_row_stride, float scale, int window, int tokens,
                                                 int H, int Hk, int D, int S, int dtype, int Dv, int keep_first,
                                                 float bias_exp, const float* sinks, int gate_col, float softcap,
                                                 int v_stride, int v_share, int out_f32, int chunk, cudaStream_t stream) {
    if (tokens <= 0) return VX_OK;
    if (Dv <= 0) Dv = D;
    if (v_stride <= 0) v_stride = Dv;
    if (v_share <= 0) v_share = 1;
    if (Hk % v_share) return VX_ERR_SHAPE;
    if (v_stride < Dv || softcap < 0.f) return VX_ERR_SHAPE;
    if (H <= 0 || Hk <= 0 || H % Hk || D <= 0 || D > ATT_MAX_D || Dv > ATT_MAX_D || S <= 0 || max_blocks <= 0)
        return VX_ERR_SHAPE;
    if (window < 0 || keep_first < 0 || bias_exp < 0.f || chunk < 0 || (chunk && keep_first)) return VX_ERR_SHAPE;
    dim3 grid(tokens, H);
    if (dtype == VX_F32)
        VX_LAUNCH_K(VX_K_ATTENTION, (paged_attention_generic_kernel<float>), grid, ATT_WARPS * 32, 0, stream, (const float*)q, q_row_stride, (const float*)k_pool, (const float*)v_pool, block_table,
            max_blocks, seq_of_token, positions, (float*)out, out_row_stride, scale, window, H, Hk, D, S, Dv, keep_first, bias_exp, sinks, gate_col, softcap, v_stride, v_share, out_f32, chunk);
    else if (dtype == VX_BF16)
        VX_LAUNCH_K(VX_K_ATTENTION, (paged_attention_generic_kernel<bf16>), grid, ATT_WARPS * 32, 0, stream, (const bf16*)q, q_row_stride, (const bf16*)k_pool, (const bf16*)v_pool, block_table,
            max_blocks, seq_of_token, positions, (bf16*)out, out_row_stride, scale, window, H, Hk, D, S, Dv, keep_first, bias_exp, sinks, gate_col, softcap, v_stride, v_share, out_f32, chunk);
    else
        return VX_ERR_DTYPE;
    VX_LAUNCH_CHECK();
    return VX_OK;
}

extern "C" int vx_paged_attention_generic_shared(const void* q, int q_row_stride, const void* k_pool,
                                                 const void* v_pool, const int* block_table, int max_blocks,
                                                 const int* seq_of_token, const int* positions, void* out,
                                                 int out_row_stride, float scale, int window, int tokens,
                                                 int H, int Hk, int D, int S, int dtype, int Dv, int keep_first,
                                                 float bias_exp, const float* sinks, int gate_col, float softcap,
                                                 int v_stride, int v_share, int out_f32, cudaStream_t stream) {
    return vx_paged_attention_generic_chunk(q, q_row_stride, k_pool, v_pool, block_table, max_blocks, seq_of_token, positions,
                                            out, out_row_stride, scale, window, tokens, H, Hk, D, S, dtype, Dv, keep_first,
                                            bias_exp, sinks, gate_col, softcap, v_stride, v_share, out_f32, 0, stream);
}

extern "C" int vx_paged_attention_generic_cap(const void* q, int q_row_stride, const void* k_pool,
                                              const void* v_pool, const int* block_table, int max_blocks,
                                              const int* seq_of_token, const int* positions, void* out,
                                              int out_row_stride, float scale, int window, int tokens,
                                              int H, int Hk, int D, int S, int dtype, int Dv, int keep_first,
                                              float bias_exp, const float* sinks, int gate_col, float softcap,
                                              int v_stride, cudaStream_t stream) {
    return vx_paged_attention_generic_shared(q, q_row_stride, k_pool, v_pool, block_table, max_blocks, seq_of_token, positions,
                                             out, out_row_stride, scale, window, tokens, H, Hk, D, S, dtype, Dv, keep_first,
                                             bias_exp, sinks, gate_col, softcap, v_stride, 1, 0, stream);
}

extern "C" int vx_paged_attention_generic(const void* q, int q_row_stride, const void* k_pool,
                                          const void* v_pool, const int* block_table, int max_blocks,
                                          const int* seq_of_token, const int* positions, void* out,
                                          int out_row_stride, float scale, int window, int tokens,
                                          int H, int Hk, int D, int S, int dtype, int Dv, int keep_first,
                                          float bias_exp, const float* sinks, int gate_col, cudaStream_t stream) {
    return vx_paged_attention_generic_cap(q, q_row_stride, k_pool, v_pool, block_table, max_blocks, seq_of_token, positions,
                                          out, out_row_stride, scale, window, tokens, H, Hk, D, S, dtype, Dv, keep_first,
                                          bias_exp, sinks, gate_col, 0.f, 0, stream);
}
