// Plain paged attention: the reference kernel that every faster attention kernel is checked
// against, and the kernel of the float32 path.  One warp per (token, query head); keys are
// walked one by one through the block table with an online softmax in float.
//
// Rule (v3/kernels/paged_attention_sm89.cu:241-369 of the reference): the q_len tokens a
// sequence brings to a step are the tail of its ctx_len cached tokens.  The token with
// in-step index i sits at position p = ctx_len - q_len + i and sees keys [0, p]; with a
// window of W keys it sees (p - W, p].  kv_head = head * nkv / nh.  A decoded token is the
// case q_len = 1.  ctx_len <= 0 marks a padded row: zeros are written, no table is read.
//
// Options for mixers that want them: `softcap` > 0 replaces a scaled score s by
// softcap * tanh(s / softcap); `sinks` (one float per query head) adds exp(sink_h) to the softmax
// denominator - a key without a value, neither scaled nor capped; `gate` (float [tokens, heads])
// multiplies each head's output; `dist` (float [nkv, dist_n, nh / nkv]) is added to a (scaled, capped) score by the distance
// between query and key, a distance beyond the last reading the last.
//
// Cache layer layout: [num_pages, planes, nkv, page_size, hd].  planes = 2: keys in plane 0, values in plane 1.
// planes = 1: one row per token and kv head; the key is the whole row and the value its leading `vd` elements
// (a latent that keys and values are projections of).  The output row of a head has `vd` elements (hd with two planes).
#include "common.cuh"

// MAX_DIMS_PER_LANE: elements of a row that one lane holds (row <= 32 * MAX_DIMS_PER_LANE; the launcher picks 8 or 32)
template <typename T, int MAX_DIMS_PER_LANE>
__global__ void paged_attention_ref_kernel(const T* __restrict__ q, const T* __restrict__ cache,
                                           const int* __restrict__ block_tables, const int* __restrict__ cu_seqlens,
                                           const int* __restrict__ ctx_lens, const int* __restrict__ token_seq,
                                           T* __restrict__ out, int n_tokens, int nh, int nkv, int hd,
                                           int page_size, int max_blocks, float scale, int window,
                                           float softcap, const float* __restrict__ sinks, const float* __restrict__ gate,
                                           int planes, int vd, const float* __restrict__ dist, int dist_n) {
    rv_pdl_launch_dependents();
    rv_pdl_wait();
    const int lane = threadIdx.x & 31;
    const int warp = threadIdx.x >> 5;
    const int t = blockIdx.x;
    const int h = blockIdx.y * (blockDim.x >> 5) + warp;
    if (h >= nh || t >= n_tokens) return;
    const int seq = token_seq[t];
    T* o = out + ((size_t)t * nh + h) * vd;
    const int ctx = seq >= 0 ? ctx_lens[seq] : 0;
    if (ctx <= 0) {
        for (int d = lane; d < vd; d += 32) o[d] = rv_from_float<T>(0.f);
        return;
    }
    const int q_start = cu_seqlens[seq];
    const int q_len = cu_seqlens[seq + 1] - q_start;
    const int pos = ctx - q_len + (t - q_start);
    const int lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
    const int kvh = (int)(((long long)h * nkv) / nh);

    float qv[MAX_DIMS_PER_LANE], acc[MAX_DIMS_PER_LANE];
    const T* qp = q + ((size_t)t * nh + h) * hd;
#pragma unroll
    for (int i = 0; i < MAX_DIMS_PER_LANE; ++i) {
        const int d = lane + 32 * i;
        qv[i] = d < hd ? rv_to_float(qp[d]) * scale : 0.f;
        acc[i] = 0.f;
    }
    float m = -INFINITY, l = 0.f;
    const int* table = block_tables + (size_t)seq * max_blocks;
    const int G = nh / nkv;
    const float* bias = dist ? dist + (size_t)kvh * dist_n * G + (h - kvh * G) : nullptr;
    const size_t page_stride = (size_t)planes * nkv * page_size * hd;
    const size_t v_off = planes == 2 ? (size_t)nkv * page_size * hd : 0;
    for (int j = lo; j <= pos; ++j) {
        const int page = table[j / page_size];
        const T* kp = cache + (size_t)page * page_stride + ((size_t)kvh * page_size + (j % page_size)) * hd;
        const T* vp = kp + v_off;
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < MAX_DIMS_PER_LANE; ++i) {
            const int d = lane + 32 * i;
            if (d < hd) s = fmaf(qv[i], rv_to_float(kp[d]), s);
        }
        s = rv_warp_sum(s);
        if (softcap > 0.f) s = softcap * tanhf(s / softcap);
        if (bias) s += bias[(size_t)min(pos - j, dist_n - 1) * G];
        const float m_new = fmaxf(m, s);
        const float corr = expf(m - m_new);     // exp(-inf) = 0 at the first key
        const float p = expf(s - m_new);
        l = l * corr + p;
#pragma unroll
        for (int i = 0; i < MAX_DIMS_PER_LANE; ++i) {
            const int d = lane + 32 * i;
            if (d < vd) acc[i] = acc[i] * corr + p * rv_to_float(vp[d]);
        }
        m = m_new;
    }
    if (sinks) {
        const float sk = sinks[h];
        const float m_new = fmaxf(m, sk);
        const float corr = expf(m - m_new);
        l = l * corr + expf(sk - m_new);
#pragma unroll
        for (int i = 0; i < MAX_DIMS_PER_LANE; ++i) acc[i] *= corr;
    }
    float inv = l > 0.f ? 1.0f / l : 0.f;
    if (gate) inv *= gate[(size_t)t * nh + h];
#pragma unroll
    for (int i = 0; i < MAX_DIMS_PER_LANE; ++i) {
        const int d = lane + 32 * i;
        if (d < vd) o[d] = rv_from_float<T>(acc[i] * inv);
    }
}

template <int DPL>
static int launch_ref(const void* q, const void* cache, const int* block_tables, const int* cu_seqlens, const int* ctx_lens,
                      const int* token_seq, void* out, int n_tokens, int nh, int nkv, int hd, int page_size, int max_blocks,
                      float scale, int window, float softcap, const float* sinks, const float* gate, int planes, int vd,
                      int dtype, const float* dist, int dist_n, cudaStream_t stream) {
    const int warps = 4;
    const dim3 grid(n_tokens, (nh + warps - 1) / warps);
    if (dtype == RV_DTYPE_F32)
        RV_LAUNCH_ST = rv_launch(paged_attention_ref_kernel<float, DPL>, dim3(grid), dim3(warps * 32), 0, stream,
            (const float*)q, (const float*)cache, block_tables, cu_seqlens, ctx_lens, token_seq, (float*)out,
            n_tokens, nh, nkv, hd, page_size, max_blocks, scale, window, softcap, sinks, gate, planes, vd, dist, dist_n);
    else if (dtype == RV_DTYPE_BF16)
        RV_LAUNCH_ST = rv_launch(paged_attention_ref_kernel<__nv_bfloat16, DPL>, dim3(grid), dim3(warps * 32), 0, stream,
            (const __nv_bfloat16*)q, (const __nv_bfloat16*)cache, block_tables, cu_seqlens, ctx_lens, token_seq,
            (__nv_bfloat16*)out, n_tokens, nh, nkv, hd, page_size, max_blocks, scale, window, softcap, sinks, gate, planes, vd, dist, dist_n);
    else
        return RV_ERR_BAD_DTYPE;
    return rv_launch_status();
}

// planes 2: keys and values in their planes, output rows of hd; planes 1: the value is the leading vd elements of the key row.
RV_EXPORT int rv_paged_attention_ref_ex(const void* q, const void* cache, const int* block_tables,
                                        const int* cu_seqlens, const int* ctx_lens, const int* token_seq,
                                        void* out, int n_tokens, int nh, int nkv, int hd, int page_size,
                                        int max_blocks, float scale, int window, float softcap, const float* sinks,
                                        const float* gate, int planes, int vd, int dtype, const float* dist, int dist_n,
                                        cudaStream_t stream) {
    if (dist && (dist_n <= 0 || nkv <= 0 || nh % nkv)) return RV_ERR_BAD_SIZE;
    if (n_tokens < 0 || nh <= 0 || nkv <= 0 || hd <= 0 || page_size <= 0 || max_blocks <= 0) return RV_ERR_BAD_SIZE;
    if ((planes != 1 && planes != 2) || vd <= 0 || vd > hd || (planes == 2 && vd != hd)) return RV_ERR_BAD_SIZE;
    if (hd > 32 * 32) return RV_ERR_UNSUPPORTED;
    if (n_tokens == 0) return RV_OK;
    if (hd <= 32 * 8)
        return launch_ref<8>(q, cache, block_tables, cu_seqlens, ctx_lens, token_seq, out, n_tokens, nh, nkv, hd, page_size,
                             max_blocks, scale, window, softcap, sinks, gate, planes, vd, dtype, dist, dist_n, stream);
    return launch_ref<32>(q, cache, block_tables, cu_seqlens, ctx_lens, token_seq, out, n_tokens, nh, nkv, hd, page_size,
                          max_blocks, scale, window, softcap, sinks, gate, planes, vd, dtype, dist, dist_n, stream);
}

RV_EXPORT int rv_paged_attention_ref(const void* q, const void* cache, const int* block_tables,
                                     const int* cu_seqlens, const int* ctx_lens, const int* token_seq,
                                     void* out, int n_tokens, int nh, int nkv, int hd, int page_size,
                                     int max_blocks, float scale, int window, float softcap, const float* sinks,
                                     const float* gate, int dtype, cudaStream_t stream) {
    if (hd > 32 * 8) return RV_ERR_UNSUPPORTED;
    return rv_paged_attention_ref_ex(q, cache, block_tables, cu_seqlens, ctx_lens, token_seq, out, n_tokens, nh, nkv, hd,
                                     page_size, max_blocks, scale, window, softcap, sinks, gate, 2, hd, dtype, nullptr, 0, stream);
}
