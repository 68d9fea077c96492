// What stands around the attention kernels for mixers whose queries and keys are rotated and then, optionally, made
// unit-RMS vectors per head, whose heads may carry two maps, and whose values may turn with their position:
//
//   qk_prepare        rows [q: nh x M x d | k: nkv x M x d | v: nkv x vd | gate logits: nh] of a float32 projection (k and v
//                     only where the layer has them; M = 1 or 2 maps per head), plus a bias per column (optional).  The
//                     leading `rot` elements of every map of q and k turn by the angle of (position, pair): pairs
//                     (2i, 2i + 1), or (i, i + rot / 2) with `halves`; with `unit` the map is then divided by
//                     sqrt(mean(x^2) + eps) over its d elements (no weight).  With value tables the value turns too, over all
//                     its vd elements in the same layout of pairs.  q goes to q_out [T, nh, M, P], k and v into the token's
//                     cache slot (planes 0 and 1 of [pages, 2, nkv, page, P]); P >= max(M d, vd).  A query row of map m holds
//                     its d elements at m d, a key row all maps side by side, so that (query row of map m) . (key row) is
//                     map m's score; everything else of a row is written as zeros.  sigmoid of the gate logits goes to a
//                     float array.  A token with slot -1 writes no key and no value.
//                     Options: weighted norms instead of the unit norm, x / sqrt(mean(x^2) + eps) * gamma IN FRONT of the
//                     rotation (one gamma of d elements for the queries, one for the keys); a factor
//                     1 + coef ln(floor((p + 1) / every) + 1) on the query of position p; the value as projected kept in a
//                     float array, or (1 - lambda) of the value plus lambda of such an array's row
//   turn_back         rows of attention results [T, nh, P]: the leading vd elements of every head turned by MINUS the token's
//                     angle, written as [T, nh, vd]
//   gate_elements     rows of attention results [T, nh, P]: the leading vd elements of every head times the sigmoid of a float
//                     logit of their own, written as [T, nh, vd]
//   map_difference    rows [T, nh, 2, P] of two maps' results: o = a1 - lambda a2 over the leading vd elements, then
//                     o / sqrt(mean(o^2) + eps) * factor, written as [T, nh, vd]
//
// All arithmetic is float; the results are rounded once, when they are stored (float or bfloat16).
#include "common.cuh"
#include <initializer_list>

#define QP_WARPS 8
#define QP_MAX_DIM 1024

__device__ __forceinline__ void qp_store(void* p, int dtype, size_t i, float v) {
    if (dtype == RV_DTYPE_F32) ((float*)p)[i] = v;
    else ((__nv_bfloat16*)p)[i] = __float2bfloat16_rn(v);
}

// V neighbouring elements per thread and access: 4 (8 or 16 bytes) where sizes and pointers allow, else 1.
template <int V>
__device__ __forceinline__ void qp_load_vec(const void* p, int dtype, size_t i, float (&v)[V]) {
    if constexpr (V == 4) {
        if (dtype == RV_DTYPE_F32) {
            const float4 f = *reinterpret_cast<const float4*>((const float*)p + i);
            v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
        } else {
            const uint2 u = *reinterpret_cast<const uint2*>((const __nv_bfloat16*)p + i);
            const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
            const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
            v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
        }
    } else {
        v[0] = dtype == RV_DTYPE_F32 ? ((const float*)p)[i] : __bfloat162float(((const __nv_bfloat16*)p)[i]);
    }
}
template <int V>
__device__ __forceinline__ void qp_store_vec(void* p, int dtype, size_t i, const float (&v)[V]) {
    if constexpr (V == 4) {
        if (dtype == RV_DTYPE_F32) {
            *reinterpret_cast<float4*>((float*)p + i) = make_float4(v[0], v[1], v[2], v[3]);
        } else {
            __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
            uint2 u;
            u.x = *reinterpret_cast<uint32_t*>(&lo); u.y = *reinterpret_cast<uint32_t*>(&hi);
            *reinterpret_cast<uint2*>((__nv_bfloat16*)p + i) = u;
        }
    } else {
        qp_store(p, dtype, i, v[0]);
    }
}

struct QkPrepareArgs {
    const float* proj; int row_stride;
    const float* bias;                                          // one per column of q, k and v, or null
    const int* positions; const float *cos_t, *sin_t; int rot, table_rows, halves;
    const float *vcos_t, *vsin_t; int v_table_rows;            // value tables [rows, vd / 2] or null
    const int* slot_mapping; void *cache, *q_out; int out_dtype; float* gate_out;
    int nh, nkv, d, vd, P, maps, page_size; float eps; int unit, write_kv;
    const float *q_gamma, *k_gamma;                             // [d] each: weighted norms in front of the rotation, or null
    float temp_coef; int temp_every;                            // temp_every 0: no temperature
    float* keep_v; const float* mix_v; float lambda;            // [T, nkv x vd] each, or null
};

// Element e of a vector of which the leading `rot` elements turn; `cs` and `sn` are the token's rows of the tables.
__device__ __forceinline__ float qp_turned(const float* v, int e, int rot, int halves, const float* __restrict__ cs,
                                           const float* __restrict__ sn) {
    const float x = v[e];
    if (e >= rot) return x;
    if (halves) {
        const int half = rot >> 1;
        const bool first = e < half;
        const int p = first ? e : e - half;
        const float other = v[first ? e + half : e - half];
        return first ? x * cs[p] - other * sn[p] : x * cs[p] + other * sn[p];
    }
    const int p = e >> 1;
    const float other = v[e ^ 1];
    return (e & 1) ? x * cs[p] + other * sn[p] : x * cs[p] - other * sn[p];
}

// One block per token; a warp takes one map of a head of q or k, or one head of v, at a time.  NJ: elements of a head slot
// per lane (P <= 32 NJ).
template <int NJ>
__global__ void __launch_bounds__(QP_WARPS * 32)
qk_prepare_kernel(const QkPrepareArgs a) {
    rv_pdl_launch_dependents();
    rv_pdl_wait();
    __shared__ float buf[QP_WARPS][32 * NJ];
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const size_t row = (size_t)t * a.row_stride;
    int pos = a.positions[t];
    if (pos < 0) pos = 0;
    const int qk_pos = pos < a.table_rows ? pos : a.table_rows - 1;      // the host refuses such positions; never read outside
    const int v_pos = pos < a.v_table_rows ? pos : a.v_table_rows - 1;
    const float* cs = a.cos_t ? a.cos_t + (size_t)qk_pos * (a.rot >> 1) : nullptr;
    const float* sn = a.sin_t ? a.sin_t + (size_t)qk_pos * (a.rot >> 1) : nullptr;
    const float* vcs = a.vcos_t ? a.vcos_t + (size_t)v_pos * (a.vd >> 1) : nullptr;
    const float* vsn = a.vcos_t ? a.vsin_t + (size_t)v_pos * (a.vd >> 1) : nullptr;
    const int slot = a.write_kv ? a.slot_mapping[t] : -1;
    const int nq = a.nh * a.maps, nk = a.nkv * a.maps;
    const int items = nq + (a.write_kv ? nk + a.nkv : 0);
    float* mine = buf[warp];
    for (int item = warp; item < items; item += QP_WARPS) {
        const int kind = item < nq ? 0 : (item < nq + nk ? 1 : 2);            // q, k, v
        const int index = kind == 0 ? item : (kind == 1 ? item - nq : item - nq - nk);
        if (kind != 0 && slot < 0 && !(kind == 2 && a.keep_v)) continue;      // (the same for the whole warp)
        const int n = kind == 2 ? a.vd : a.d;
        const int head = kind == 2 ? index : index / a.maps, map = kind == 2 ? 0 : index - head * a.maps;
        const size_t col = kind == 0 ? (size_t)index * a.d
                                     : (kind == 1 ? (size_t)(nq + index) * a.d : (size_t)(nq + nk) * a.d + (size_t)index * a.vd);
        const float* gamma = kind == 0 ? a.q_gamma : (kind == 1 ? a.k_gamma : nullptr);
        float before = 0.f;
        for (int i = lane; i < n; i += 32) {
            float v = a.proj[row + col + i] + (a.bias ? a.bias[col + i] : 0.f);
            if (kind == 2) {
                const size_t at = ((size_t)t * a.nkv + index) * a.vd + i;
                if (a.keep_v) a.keep_v[at] = v;
                if (a.mix_v) v = (1.0f - a.lambda) * v + a.lambda * a.mix_v[at];
            }
            mine[i] = v;
            before = fmaf(v, v, before);
        }
        if (kind != 0 && slot < 0) continue;
        if (gamma) {                                                          // a lane scales what it has stored itself
            const float g = 1.0f / sqrtf(rv_warp_sum(before) / (float)n + a.eps);
            for (int i = lane; i < n; i += 32) mine[i] = mine[i] * g * gamma[i];
        }
        __syncwarp();
        const float* c = kind == 2 ? vcs : cs;
        const float* s = kind == 2 ? vsn : sn;
        const int rot = c ? (kind == 2 ? a.vd : a.rot) : 0;
        const int at = map * a.d;                                             // where the map lies in its row
        float vals[NJ];
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const int e = lane + 32 * j - at;
            const float v = (e >= 0 && e < n) ? qp_turned(mine, e, rot, a.halves, c, s) : 0.f;
            vals[j] = v;
            ss = fmaf(v, v, ss);
        }
        float r = 1.f;
        if (kind != 2 && a.unit) {
            ss = rv_warp_sum(ss);
            r = 1.0f / sqrtf(ss / (float)n + a.eps);
        }
        if (kind == 0 && a.temp_every > 0) r *= 1.0f + a.temp_coef * logf((float)((pos + 1) / a.temp_every + 1));
        void* dst_base;
        size_t dst;
        if (kind == 0) {
            dst_base = a.q_out;
            dst = ((size_t)t * nq + index) * a.P;
        } else {
            dst_base = a.cache;
            const size_t page = (size_t)(slot / a.page_size), off = (size_t)(slot % a.page_size);
            dst = (((page * 2 + (kind == 2 ? 1 : 0)) * a.nkv + head) * a.page_size + off) * a.P;
        }
        // a key's maps are written by different warps: each its own elements, the last one the row's tail as well
        const int lo = kind == 1 ? at : 0, hi = (kind == 1 && map + 1 < a.maps) ? at + a.d : a.P;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const int i = lane + 32 * j;
            if (i >= lo && i < hi) qp_store(dst_base, a.out_dtype, dst + i, vals[j] * r);
        }
        __syncwarp();
    }
    if (a.gate_out) {
        const size_t g0 = row + (size_t)nq * a.d + (a.write_kv ? (size_t)nk * a.d + (size_t)a.nkv * a.vd : 0);
        for (int h = threadIdx.x; h < a.nh; h += blockDim.x)
            a.gate_out[(size_t)t * a.nh + h] = 1.0f / (1.0f + expf(-a.proj[g0 + h]));
    }
}

// The same for one map per head whose pairs, if any, are neighbours, with sizes in multiples of 4: a warp per (token, head of q, k
// or v), a lane holds four neighbouring elements per step (pairs never leave a lane), nothing passes through shared memory.  NJ:
// steps (P <= 128 NJ).  Item `items` of a token is its gate logits.
template <int NJ>
__global__ void __launch_bounds__(QP_WARPS * 32)
qk_prepare_vec_kernel(const QkPrepareArgs a, int items, int per_token, size_t total) {
    rv_pdl_launch_dependents();
    rv_pdl_wait();
    const int lane = threadIdx.x & 31;
    const size_t w = (size_t)blockIdx.x * QP_WARPS + (threadIdx.x >> 5);
    if (w >= total) return;
    const size_t t = w / per_token;
    const int item = (int)(w - t * per_token);
    const size_t row = t * a.row_stride;
    if (item >= items) {
        const size_t g0 = row + (size_t)a.nh * a.d + (a.write_kv ? (size_t)a.nkv * (a.d + a.vd) : 0);
        for (int h = lane; h < a.nh; h += 32) a.gate_out[t * a.nh + h] = 1.0f / (1.0f + expf(-a.proj[g0 + h]));
        return;
    }
    const int kind = item < a.nh ? 0 : (item < a.nh + a.nkv ? 1 : 2);               // q, k, v
    const int index = kind == 0 ? item : (kind == 1 ? item - a.nh : item - a.nh - a.nkv);
    const int n = kind == 2 ? a.vd : a.d;
    const size_t col = kind == 2 ? (size_t)(a.nh + a.nkv) * a.d + (size_t)index * a.vd : (size_t)item * a.d;
    int pos = a.positions[t];
    if (pos < 0) pos = 0;
    const int slot = kind == 0 ? 0 : a.slot_mapping[t];
    const float* cos_t = kind == 2 ? a.vcos_t : a.cos_t;
    const float* sin_t = kind == 2 ? a.vsin_t : a.sin_t;
    const int rot = cos_t ? (kind == 2 ? a.vd : a.rot) : 0, rows = kind == 2 ? a.v_table_rows : a.table_rows;
    const size_t tab = (size_t)(pos < rows ? pos : rows - 1) * (rot >> 1);          // the host refuses such positions; never read outside
    const float* gamma = kind == 0 ? a.q_gamma : (kind == 1 ? a.k_gamma : nullptr);
    float v[NJ][4];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        const int e = (lane + 32 * j) * 4;
        v[j][0] = v[j][1] = v[j][2] = v[j][3] = 0.f;
        if (e < n) {
            qp_load_vec<4>(a.proj, RV_DTYPE_F32, row + col + e, v[j]);
            if (a.bias) {
                float b[4];
                qp_load_vec<4>(a.bias, RV_DTYPE_F32, col + e, b);
#pragma unroll
                for (int i = 0; i < 4; ++i) v[j][i] += b[i];
            }
            if (kind == 2) {
                const size_t at = (t * a.nkv + index) * a.vd + e;
                if (a.keep_v) qp_store_vec<4>(a.keep_v, RV_DTYPE_F32, at, v[j]);
                if (a.mix_v) {
                    float f[4];
                    qp_load_vec<4>(a.mix_v, RV_DTYPE_F32, at, f);
#pragma unroll
                    for (int i = 0; i < 4; ++i) v[j][i] = (1.0f - a.lambda) * v[j][i] + a.lambda * f[i];
                }
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) ss = fmaf(v[j][i], v[j][i], ss);                // (a turn leaves the sum as it is)
    }
    if (slot < 0) return;
    float r = 1.f;
    if (kind != 2 && (gamma || a.unit)) r = 1.0f / sqrtf(rv_warp_sum(ss) / (float)n + a.eps);
    float post = 1.f;                                                               // behind the norm's weight
    if (kind == 0 && a.temp_every > 0) post = 1.0f + a.temp_coef * logf((float)((pos + 1) / a.temp_every + 1));
    void* dst_base = kind == 0 ? a.q_out : a.cache;
    const size_t page = (size_t)(slot / a.page_size), off = (size_t)(slot % a.page_size);
    const size_t dst = kind == 0 ? (t * a.nh + index) * a.P
                                 : (((page * 2 + (kind == 2 ? 1 : 0)) * a.nkv + index) * a.page_size + off) * a.P;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        const int e = (lane + 32 * j) * 4;
        if (e >= a.P) continue;
        if (e < n) {
            float g[4] = {1.f, 1.f, 1.f, 1.f};
            if (gamma) qp_load_vec<4>(gamma, RV_DTYPE_F32, e, g);
#pragma unroll
            for (int i = 0; i < 4; ++i) v[j][i] = v[j][i] * r * g[i];
#pragma unroll
            for (int i = 0; i < 4; i += 2) {
                if (e + i < rot) {
                    const float c = cos_t[tab + ((e + i) >> 1)], s = sin_t[tab + ((e + i) >> 1)];
                    const float x = v[j][i], y = v[j][i + 1];
                    v[j][i] = x * c - y * s;
                    v[j][i + 1] = y * c + x * s;
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) v[j][i] *= post;
        }
        qp_store_vec<4>(dst_base, a.out_dtype, dst + e, v[j]);
    }
}

// q_gamma and k_gamma go together and exclude `unit`; keep_v and mix_v are float [n_tokens, nkv * vd].
RV_EXPORT int rv_qk_prepare_ex(const float* proj, int row_stride, const float* bias, const int* positions, const float* cos_t,
                               const float* sin_t, int rot, int table_rows, int halves, const float* vcos_t, const float* vsin_t,
                               int v_table_rows, const int* slot_mapping, void* cache, void* q_out, int out_dtype, float* gate_out,
                               int n_tokens, int nh, int nkv, int d, int vd, int P, int maps, int page_size, float eps, int unit,
                               int write_kv, const float* q_gamma, const float* k_gamma, float temp_coef, int temp_every,
                               float* keep_v, const float* mix_v, float lambda, cudaStream_t stream) {
    if ((q_gamma == nullptr) != (k_gamma == nullptr) || (q_gamma && unit) || temp_every < 0) return RV_ERR_BAD_SIZE;
    if ((keep_v || mix_v) && !write_kv) return RV_ERR_BAD_SIZE;
    if (n_tokens < 0 || nh <= 0 || nkv <= 0 || d <= 0 || vd <= 0 || P < vd || page_size <= 0 || table_rows <= 0 || v_table_rows <= 0)
        return RV_ERR_BAD_SIZE;
    if (maps != 1 && maps != 2) return RV_ERR_BAD_SIZE;
    if (P > QP_MAX_DIM || d > QP_MAX_DIM) return RV_ERR_UNSUPPORTED;
    if (P < maps * d) return RV_ERR_BAD_SIZE;
    if (rot < 0 || rot > d || (rot & 1)) return RV_ERR_BAD_SIZE;
    if ((vcos_t == nullptr) != (vsin_t == nullptr) || (vcos_t && (vd & 1))) return RV_ERR_BAD_SIZE;
    if (row_stride < maps * nh * d + (write_kv ? nkv * (maps * d + vd) : 0) + (gate_out ? nh : 0)) return RV_ERR_BAD_SIZE;
    if (write_kv && (!slot_mapping || !cache)) return RV_ERR_BAD_SIZE;
    if (out_dtype & ~1) return RV_ERR_BAD_DTYPE;
    if (n_tokens == 0) return RV_OK;
    if (!cos_t || !sin_t) { cos_t = sin_t = nullptr; rot = 0; }
    const QkPrepareArgs a = {proj, row_stride, bias, positions, cos_t, sin_t, rot, table_rows, halves, vcos_t, vsin_t, v_table_rows,
                             slot_mapping, cache, q_out, out_dtype, gate_out, nh, nkv, d, vd, P, maps, page_size, eps, unit, write_kv,
                             q_gamma, k_gamma, temp_coef, temp_every, keep_v, mix_v, lambda};
    uintptr_t bits = 0;
    for (const void* p : {(const void*)proj, (const void*)bias, (const void*)cache, (const void*)q_out, (const void*)q_gamma, (const void*)k_gamma,
                          (const void*)keep_v, (const void*)mix_v})
        bits |= reinterpret_cast<uintptr_t>(p);
    if (maps == 1 && (!halves || (rot == 0 && !vcos_t)) && d % 4 == 0 && vd % 4 == 0 && P % 4 == 0 && row_stride % 4 == 0 && bits % 16 == 0) {
        const int items = nh + (write_kv ? 2 * nkv : 0), per_token = items + (gate_out ? 1 : 0);
        const size_t total = (size_t)n_tokens * per_token, blocks = (total + QP_WARPS - 1) / QP_WARPS;
        if (blocks <= 0x7fffffffULL) {
            auto vec = P <= 128 ? qk_prepare_vec_kernel<1> : (P <= 256 ? qk_prepare_vec_kernel<2> : qk_prepare_vec_kernel<8>);
            RV_LAUNCH_ST = rv_launch(vec, dim3((unsigned)blocks), dim3(QP_WARPS * 32), 0, stream, a, items, per_token, total);
            return rv_launch_status();
        }
    }
    auto kernel = P <= 32 ? qk_prepare_kernel<1> : (P <= 64 ? qk_prepare_kernel<2> : (P <= 128 ? qk_prepare_kernel<4>
                : (P <= 256 ? qk_prepare_kernel<8> : qk_prepare_kernel<32>)));
    RV_LAUNCH_ST = rv_launch(kernel, dim3(n_tokens), dim3(QP_WARPS * 32), 0, stream, a);
    return rv_launch_status();
}

RV_EXPORT int rv_qk_prepare(const float* proj, int row_stride, const float* bias, const int* positions, const float* cos_t,
                            const float* sin_t, int rot, int table_rows, int halves, const float* vcos_t, const float* vsin_t,
                            int v_table_rows, const int* slot_mapping, void* cache, void* q_out, int out_dtype, float* gate_out,
                            int n_tokens, int nh, int nkv, int d, int vd, int P, int maps, int page_size, float eps, int unit,
                            int write_kv, cudaStream_t stream) {
    return rv_qk_prepare_ex(proj, row_stride, bias, positions, cos_t, sin_t, rot, table_rows, halves, vcos_t, vsin_t, v_table_rows,
                            slot_mapping, cache, q_out, out_dtype, gate_out, n_tokens, nh, nkv, d, vd, P, maps, page_size, eps, unit,
                            write_kv, nullptr, nullptr, 0.f, 0, nullptr, nullptr, 0.f, stream);
}

// ------------------------------------------------------------------ after the attention kernels
// A thread takes V neighbouring pairs.  halves: pairs (m, m + vd / 2); else (2m, 2m + 1), V = 1.
template <int V>
__global__ void __launch_bounds__(256)
turn_back_kernel(const void* __restrict__ o, const int* __restrict__ positions, const float* __restrict__ cos_t,
                 const float* __restrict__ sin_t, int table_rows, int halves, void* __restrict__ out, int dtype, int nh, int vd, int P,
                 size_t total) {
    rv_pdl_launch_dependents();
    rv_pdl_wait();
    const int half = vd >> 1, per_head = half / V, per_token = per_head * nh;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const size_t t = i / per_token;
        const int in_token = (int)(i - t * per_token), h = in_token / per_head, m = (in_token - h * per_head) * V;
        int pos = positions[t];
        if (pos < 0) pos = 0;
        if (pos >= table_rows) pos = table_rows - 1;
        const size_t src = (t * nh + h) * P, dst = (t * nh + h) * vd;
        const int first = halves ? m : 2 * m, second = halves ? m + half : 2 * m + 1;
        float a[V], b[V], c[V], s[V], u[V], w[V];
        qp_load_vec<V>(o, dtype, src + first, a);
        qp_load_vec<V>(o, dtype, src + second, b);
        qp_load_vec<V>(cos_t, RV_DTYPE_F32, (size_t)pos * half + m, c);
        qp_load_vec<V>(sin_t, RV_DTYPE_F32, (size_t)pos * half + m, s);
#pragma unroll
        for (int j = 0; j < V; ++j) {
            u[j] = a[j] * c[j] + b[j] * s[j];
            w[j] = b[j] * c[j] - a[j] * s[j];
        }
        qp_store_vec<V>(out, dtype, dst + first, u);
        qp_store_vec<V>(out, dtype, dst + second, w);
    }
}

static inline int qp_blocks(size_t items) {
    const size_t want = (items + 255) / 256;
    return (int)(want < 148 * 16 ? (want ? want : 1) : 148 * 16);
}

RV_EXPORT int rv_turn_back(const void* o, const int* positions, const float* cos_t, const float* sin_t, int table_rows, int halves,
                           void* out, int dtype, int n_tokens, int nh, int vd, int P, cudaStream_t stream) {
    if (n_tokens < 0 || nh <= 0 || vd <= 0 || (vd & 1) || P < vd || table_rows <= 0) return RV_ERR_BAD_SIZE;
    if (dtype & ~1) return RV_ERR_BAD_DTYPE;
    if (n_tokens == 0) return RV_OK;
    const uintptr_t bits = reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(cos_t) |
                           reinterpret_cast<uintptr_t>(sin_t);
    const size_t pairs = (size_t)n_tokens * nh * (vd / 2);
    if (halves && vd % 8 == 0 && P % 4 == 0 && bits % 16 == 0)
        RV_LAUNCH_ST = rv_launch(turn_back_kernel<4>, dim3(qp_blocks(pairs / 4)), dim3(256), 0, stream, o, positions, cos_t, sin_t,
                                 table_rows, halves, out, dtype, nh, vd, P, pairs / 4);
    else
        RV_LAUNCH_ST = rv_launch(turn_back_kernel<1>, dim3(qp_blocks(pairs)), dim3(256), 0, stream, o, positions, cos_t, sin_t,
                                 table_rows, halves, out, dtype, nh, vd, P, pairs);
    return rv_launch_status();
}

// A thread takes V neighbouring elements of a head.
template <int V>
__global__ void __launch_bounds__(256)
gate_elements_kernel(const void* __restrict__ o, const float* __restrict__ logits, int g_stride, void* __restrict__ out, int dtype, int nh,
                     int vd, int P, size_t total) {
    rv_pdl_launch_dependents();
    rv_pdl_wait();
    const int per_head = vd / V, per_token = per_head * nh;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const size_t t = i / per_token;
        const int in_token = (int)(i - t * per_token), h = in_token / per_head, e = (in_token - h * per_head) * V;
        float v[V], g[V];
        qp_load_vec<V>(o, dtype, (t * nh + h) * P + e, v);
        qp_load_vec<V>(logits, RV_DTYPE_F32, t * g_stride + (size_t)h * vd + e, g);
#pragma unroll
        for (int j = 0; j < V; ++j) v[j] = v[j] / (1.0f + expf(-g[j]));
        qp_store_vec<V>(out, dtype, (t * nh + h) * vd + e, v);
    }
}

// logits: float rows of g_stride elements, of which the first nh * vd are the gates' (the pointer is at the first column).
RV_EXPORT int rv_gate_elements(const void* o, const float* logits, int g_stride, void* out, int dtype, int n_tokens, int nh, int vd, int P,
                               cudaStream_t stream) {
    if (n_tokens < 0 || nh <= 0 || vd <= 0 || P < vd || g_stride < nh * vd) return RV_ERR_BAD_SIZE;
    if (dtype & ~1) return RV_ERR_BAD_DTYPE;
    if (n_tokens == 0) return RV_OK;
    const uintptr_t bits = reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(logits);
    const size_t total = (size_t)n_tokens * nh * vd;
    if (vd % 4 == 0 && P % 4 == 0 && g_stride % 4 == 0 && bits % 16 == 0)
        RV_LAUNCH_ST = rv_launch(gate_elements_kernel<4>, dim3(qp_blocks(total / 4)), dim3(256), 0, stream, o, logits, g_stride, out, dtype,
                                 nh, vd, P, total / 4);
    else
        RV_LAUNCH_ST = rv_launch(gate_elements_kernel<1>, dim3(qp_blocks(total)), dim3(256), 0, stream, o, logits, g_stride, out, dtype,
                                 nh, vd, P, total);
    return rv_launch_status();
}

// One warp per (token, head); a head's vd elements in NJ accesses of V per lane (vd <= 32 V NJ).
template <int V, int NJ>
__global__ void __launch_bounds__(256)
map_difference_kernel(const void* __restrict__ o, float lambda, float eps, float factor, void* __restrict__ out, int dtype, int vd,
                      int P, size_t total_heads) {
    rv_pdl_launch_dependents();
    rv_pdl_wait();
    const int lane = threadIdx.x & 31;
    const size_t w = (size_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (w >= total_heads) return;
    const size_t first = w * 2 * P, second = first + P;
    float v[NJ][V];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        const int i = (j * 32 + lane) * V;
        if (i < vd) {
            float b[V];
            qp_load_vec<V>(o, dtype, first + i, v[j]);
            qp_load_vec<V>(o, dtype, second + i, b);
#pragma unroll
            for (int k = 0; k < V; ++k) {
                v[j][k] = fmaf(-lambda, b[k], v[j][k]);
                ss = fmaf(v[j][k], v[j][k], ss);
            }
        }
    }
    ss = rv_warp_sum(ss);
    const float r = factor / sqrtf(ss / (float)vd + eps);
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
        const int i = (j * 32 + lane) * V;
        if (i < vd) {
#pragma unroll
            for (int k = 0; k < V; ++k) v[j][k] *= r;
            qp_store_vec<V>(out, dtype, w * vd + i, v[j]);
        }
    }
}

RV_EXPORT int rv_map_difference(const void* o, float lambda, float eps, float factor, void* out, int dtype, int n_tokens, int nh, int vd,
                                int P, cudaStream_t stream) {
    if (n_tokens < 0 || nh <= 0 || vd <= 0 || P < vd) return RV_ERR_BAD_SIZE;
    if (vd > QP_MAX_DIM) return RV_ERR_UNSUPPORTED;
    if (dtype & ~1) return RV_ERR_BAD_DTYPE;
    if (n_tokens == 0) return RV_OK;
    const size_t total = (size_t)n_tokens * nh;
    const dim3 grid((unsigned)((total + 7) / 8));
    const bool vec = vd % 4 == 0 && P % 4 == 0 && ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(out)) % 16) == 0;
    auto kernel = vec ? (vd <= 128 ? map_difference_kernel<4, 1> : (vd <= 256 ? map_difference_kernel<4, 2> : map_difference_kernel<4, 8>))
                      : (vd <= 128 ? map_difference_kernel<1, 4> : (vd <= 256 ? map_difference_kernel<1, 8> : map_difference_kernel<1, 32>));
    RV_LAUNCH_ST = rv_launch(kernel, grid, dim3(256), 0, stream, o, lambda, eps, factor, out, dtype, vd, P, total);
    return rv_launch_status();
}
