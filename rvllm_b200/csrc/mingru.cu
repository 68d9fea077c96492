// minGRU: a gated recurrence whose gates read only the current token, channel by channel,
//
//   z = sigmoid(Z + bz),  u = X + bx,  c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0)
//   S <- (1 - z) S + z c;     y = S silu(G)
//
// with [Z | X | G] the columns of a float32 projection.  S is kept per request and channel in float32; y is rounded once.
//
// A step S -> a S + b is an affine map, and affine maps compose: (a2, b2) after (a1, b1) is (a1 a2, a2 b1 + b2).  So a prompt
// portion is not walked token by token: a CTA owns MG_CHANNELS channels of one sequence and takes MG_RUNS * MG_RUN tokens at a
// time.  A thread forms the maps of MG_RUN neighbouring tokens of one channel in registers and their composition; the
// compositions go through shared memory, every thread applies those of the runs before its own to the state that the tokens
// so far have left, and then applies its own maps one by one.  The next tokens' inputs are loaded before the exchange and
// wait in registers.  Sixteen channels a CTA (rows of 64 bytes) leave room for two CTAs on an SM, one of which computes while
// the other waits for its loads or its barrier.  Steps of single tokens take a kernel with a thread per channel.
//
// state [slots][channels]; a sequence with slot -1 starts from zero and leaves no state.  Nothing is read on the host.
#include "common.cuh"

#define MG_CHANNELS 16
#define MG_RUNS 32
#define MG_RUN 4
#define MG_THREADS (MG_CHANNELS * MG_RUNS)

__device__ __forceinline__ float mg_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }

__device__ __forceinline__ void mg_step(float z_raw, float x_raw, float zb, float xb, float& a, float& b) {
    const float z = mg_sigmoid(z_raw + zb), u = x_raw + xb;
    a = 1.0f - z;
    b = z * (u >= 0.f ? u + 0.5f : mg_sigmoid(u));
}

__device__ __forceinline__ void mg_store(void* out, int dtype, size_t i, float v) {
    if (dtype == RV_DTYPE_F32) ((float*)out)[i] = v;
    else ((__nv_bfloat16*)out)[i] = __float2bfloat16_rn(v);
}

// grid (channel blocks, sequences)
__global__ void __launch_bounds__(MG_THREADS, 2)
mingru_scan_kernel(const float* __restrict__ proj, int stride, const float* __restrict__ z_bias, const float* __restrict__ x_bias,
                   const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots, float* __restrict__ state,
                   long long state_stride, void* __restrict__ out, int out_dtype, int channels) {
    rv_pdl_launch_dependents();
    rv_pdl_wait();
    __shared__ float2 maps[2][MG_RUNS][MG_CHANNELS];
    const int lane = threadIdx.x % MG_CHANNELS, run = threadIdx.x / MG_CHANNELS;
    const int ch = blockIdx.x * MG_CHANNELS + lane, seq = blockIdx.y;
    const bool live = ch < channels;
    const int first = cu_seqlens[seq], end = cu_seqlens[seq + 1];
    const int slot = state_slots[seq];
    const float zb = live ? z_bias[ch] : 0.f, xb = live ? x_bias[ch] : 0.f;
    float S = (live && slot >= 0) ? state[(size_t)slot * state_stride + ch] : 0.f;
    float z[MG_RUN], x[MG_RUN], g[MG_RUN];
    auto fetch = [&](int t0) {
#pragma unroll
        for (int i = 0; i < MG_RUN; ++i) {
            const int t = t0 + i;
            const bool in = live && t < end;
            const float* p = proj + (size_t)t * stride + ch;
            z[i] = in ? __ldg(p) : 0.f;
            x[i] = in ? __ldg(p + channels) : 0.f;
            g[i] = in ? __ldg(p + 2 * channels) : 0.f;
        }
    };
    int t0 = first + run * MG_RUN;
    fetch(t0);
    for (int base = first, turn = 0; base < end; base += MG_RUNS * MG_RUN, turn ^= 1) {
        float a[MG_RUN], b[MG_RUN], gate[MG_RUN];
        float A = 1.f, B = 0.f;
#pragma unroll
        for (int i = 0; i < MG_RUN; ++i) {
            if (t0 + i < end) mg_step(z[i], x[i], zb, xb, a[i], b[i]);
            else { a[i] = 1.f; b[i] = 0.f; }                        // beyond the sequence: the map that changes nothing
            gate[i] = g[i] * mg_sigmoid(g[i]);
            A *= a[i];
            B = fmaf(a[i], B, b[i]);
        }
        const int mine = t0;
        t0 += MG_RUNS * MG_RUN;
        fetch(t0);
        maps[turn][run][lane] = make_float2(A, B);
        __syncthreads();                                            // (two places in turn: one barrier a pass is enough)
        float before = S;
#pragma unroll
        for (int w = 0; w < MG_RUNS; ++w) {
            if (w == run) before = S;
            const float2 m = maps[turn][w][lane];
            S = fmaf(m.x, S, m.y);
        }
#pragma unroll
        for (int i = 0; i < MG_RUN; ++i) {
            before = fmaf(a[i], before, b[i]);
            if (live && mine + i < end) mg_store(out, out_dtype, (size_t)(mine + i) * channels + ch, before * gate[i]);
        }
    }
    if (run == 0 && live && slot >= 0 && end > first) state[(size_t)slot * state_stride + ch] = S;
}

// one token per sequence; grid (channel blocks, sequences)
__global__ void __launch_bounds__(128)
mingru_token_kernel(const float* __restrict__ proj, int stride, const float* __restrict__ z_bias, const float* __restrict__ x_bias,
                    const int* __restrict__ state_slots, float* __restrict__ state, long long state_stride, void* __restrict__ out,
                    int out_dtype, int channels) {
    rv_pdl_launch_dependents();
    rv_pdl_wait();
    const int ch = blockIdx.x * 128 + threadIdx.x, seq = blockIdx.y;
    if (ch >= channels) return;
    const int slot = state_slots[seq];
    const float* p = proj + (size_t)seq * stride + ch;
    const float z = p[0], x = p[channels], g = p[2 * channels];
    float S = slot >= 0 ? state[(size_t)slot * state_stride + ch] : 0.f;
    float a, b;
    mg_step(z, x, z_bias[ch], x_bias[ch], a, b);
    S = fmaf(a, S, b);
    if (slot >= 0) state[(size_t)slot * state_stride + ch] = S;
    mg_store(out, out_dtype, (size_t)seq * channels + ch, S * (g * mg_sigmoid(g)));
}

// proj float rows [Z | X | G | ...] of `stride`; single: every sequence brings exactly one token (n_tokens = n_seqs).
RV_EXPORT int rv_mingru(const float* proj, int stride, const float* z_bias, const float* x_bias, const int* cu_seqlens,
                        const int* state_slots, float* state, long long state_stride, void* out, int out_dtype, int n_seqs,
                        int channels, int single, cudaStream_t stream) {
    if (n_seqs < 0 || n_seqs > 65535 || channels <= 0 || stride < 3 * channels || state_stride < channels) return RV_ERR_BAD_SIZE;
    if (out_dtype & ~1) return RV_ERR_BAD_DTYPE;
    if (n_seqs == 0) return RV_OK;
    if (single)
        RV_LAUNCH_ST = rv_launch(mingru_token_kernel, dim3((channels + 127) / 128, n_seqs), dim3(128), 0, stream, proj, stride, z_bias,
                                 x_bias, state_slots, state, state_stride, out, out_dtype, channels);
    else
        RV_LAUNCH_ST = rv_launch(mingru_scan_kernel, dim3((channels + MG_CHANNELS - 1) / MG_CHANNELS, n_seqs), dim3(MG_THREADS), 0, stream, proj, stride,
                                 z_bias, x_bias, cu_seqlens, state_slots, state, state_stride, out, out_dtype, channels);
    return rv_launch_status();
}
