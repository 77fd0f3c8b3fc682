// The norm without statistics: y = tanh(alpha * x) * w + b with one alpha, in float.
//
// Nothing is reduced, so every element stands alone and the norm fuses with whatever makes or takes its input:
//   * dynamic_tanh      out[r, :] = norm(x[rows[r], :]) in the storage type asked for (the norm in front of a sublayer);
//   * embed             out[t, :] = norm(table[ids[t], :] * scale) in float;
//   * add               residual[t, :] += mult * norm(y[t, :]) (the norm behind a sublayer), and, when the norm that reads the
//     new stream next is known, copy[t, :] = next(residual[t, :]) in the storage type asked for, in the same pass.  y is
//     a float matrix, or the weighted sum of a token's rows among experts' results plus one more row for every token (the
//     sum in the order of the choices, as the combining kernel of the experts forms it), so that sum is never written.
#include "common.cuh"

namespace {

struct Dyt { const float* w; const float* b; float alpha; };

__device__ __forceinline__ float dyt1(float x, float a, float w, float b) { return fmaf(tanhf(a * x), w, b); }
__device__ __forceinline__ float4 dyt4(float4 x, const Dyt& n, int i) {
    const float4 w = *reinterpret_cast<const float4*>(n.w + i), b = *reinterpret_cast<const float4*>(n.b + i);
    return make_float4(dyt1(x.x, n.alpha, w.x, b.x), dyt1(x.y, n.alpha, w.y, b.y), dyt1(x.z, n.alpha, w.z, b.z), dyt1(x.w, n.alpha, w.w, b.w));
}

// V elements per thread and turn (4: sizes and pointers allow 16-byte accesses)
template <typename TO, int V>
__global__ void __launch_bounds__(256)
dynamic_tanh_kernel(const float* __restrict__ x, const int* __restrict__ rows_in, Dyt n, TO* __restrict__ out, unsigned total, unsigned d) {
    ik_pdl_wait();
    IK_AFTER_WAIT(x);
    IK_AFTER_WAIT(rows_in);
    ik_pdl_launch_dependents();
    const unsigned stride = gridDim.x * blockDim.x * V;
    for (unsigned idx = (blockIdx.x * blockDim.x + threadIdx.x) * V; idx < total; idx += stride) {
        const unsigned r = idx / d, i = idx - r * d;
        const size_t src = rows_in ? (size_t)rows_in[r] * d + i : idx;
        if (V == 4) ik_st4(out, idx, dyt4(ik_ld4(x, src), n, i));
        else ik_st(out, idx, dyt1(x[src], n.alpha, n.w[i], n.b[i]));
    }
}

template <typename TW, int V>
__global__ void __launch_bounds__(256)
dynamic_tanh_embed_kernel(const int* __restrict__ ids, const TW* __restrict__ table, Dyt n, float* __restrict__ out, unsigned total, unsigned d,
                          int vocab, float scale, int* status) {
    ik_pdl_wait();
    IK_AFTER_WAIT(ids);
    ik_pdl_launch_dependents();
    const unsigned stride = gridDim.x * blockDim.x * V;
    for (unsigned idx = (blockIdx.x * blockDim.x + threadIdx.x) * V; idx < total; idx += stride) {
        const unsigned t = idx / d, i = idx - t * d;
        const int id = ids[t];
        const bool ok = id >= 0 && id < vocab;
        if (!ok && i == 0) ik_set_status(status, IK_STATUS_BAD_TOKEN);
        const size_t src = (size_t)(ok ? id : 0) * d + i;
        if (V == 4) {
            float4 v = ik_ld4(table, src);
            v.x *= scale; v.y *= scale; v.z *= scale; v.w *= scale;
            ik_st4(out, idx, ok ? dyt4(v, n, i) : make_float4(0.f, 0.f, 0.f, 0.f));
        } else {
            out[idx] = ok ? dyt1(ik_ld(table, src) * scale, n.alpha, n.w[i], n.b[i]) : 0.f;
        }
    }
}

struct Parts {                                           // the experts' results a token's y is the sum of
    const float* parts; const float* weight; const int* row_of; const float* extra; const float* extra_weight;
    int top;
};

template <typename TO, int V, bool SUM>
__global__ void __launch_bounds__(256)
dynamic_tanh_add_kernel(const float* __restrict__ y, Parts s, Dyt n, float* __restrict__ residual, float mult, Dyt next, TO* __restrict__ copy,
                        unsigned total, unsigned d) {
    ik_pdl_wait();
    IK_AFTER_WAIT(y);
    IK_AFTER_WAIT(s.parts);
    IK_AFTER_WAIT(s.weight);
    IK_AFTER_WAIT(s.row_of);
    IK_AFTER_WAIT(s.extra);
    IK_AFTER_WAIT(s.extra_weight);
    IK_AFTER_WAIT(residual);
    ik_pdl_launch_dependents();
    const unsigned stride = gridDim.x * blockDim.x * V;
    for (unsigned idx = (blockIdx.x * blockDim.x + threadIdx.x) * V; idx < total; idx += stride) {
        const unsigned t = idx / d, i = idx - t * d;
        float v[V];
        if (SUM) {
            #pragma unroll
            for (int j = 0; j < V; j++) v[j] = 0.f;
            #pragma unroll 4
            for (int k = 0; k < s.top; k++) {
                const size_t a = (size_t)t * s.top + k;
                const float wk = s.weight ? s.weight[a] : 1.0f;
                const float* src = s.parts + (s.row_of ? (size_t)s.row_of[a] : a) * d + i;
                if (V == 4) {
                    const float4 p = *reinterpret_cast<const float4*>(src);
                    v[0] = fmaf(wk, p.x, v[0]); v[1 % V] = fmaf(wk, p.y, v[1 % V]); v[2 % V] = fmaf(wk, p.z, v[2 % V]); v[3 % V] = fmaf(wk, p.w, v[3 % V]);
                } else {
                    v[0] = fmaf(wk, src[0], v[0]);
                }
            }
            if (s.extra) {
                const float we = s.extra_weight ? s.extra_weight[t] : 1.0f;
                #pragma unroll
                for (int j = 0; j < V; j++) v[j] = fmaf(we, s.extra[idx + j], v[j]);
            }
        } else if (V == 4) {
            const float4 p = *reinterpret_cast<const float4*>(y + idx);
            v[0] = p.x; v[1 % V] = p.y; v[2 % V] = p.z; v[3 % V] = p.w;
        } else {
            v[0] = y[idx];
        }
        if (V == 4) {
            float4 r = *reinterpret_cast<const float4*>(residual + idx);
            const float4 a = dyt4(make_float4(v[0], v[1 % V], v[2 % V], v[3 % V]), n, i);
            r.x = fmaf(mult, a.x, r.x); r.y = fmaf(mult, a.y, r.y); r.z = fmaf(mult, a.z, r.z); r.w = fmaf(mult, a.w, r.w);
            *reinterpret_cast<float4*>(residual + idx) = r;
            if (copy) ik_st4(copy, idx, dyt4(r, next, i));
        } else {
            const float r = fmaf(mult, dyt1(v[0], n.alpha, n.w[i], n.b[i]), residual[idx]);
            residual[idx] = r;
            if (copy) ik_st(copy, idx, dyt1(r, next.alpha, next.w[i], next.b[i]));
        }
    }
}

inline int blocks_for(unsigned turns) {
    const unsigned want = (turns + 255) / 256, cap = (unsigned)ik_sm_count() * 16;
    return (int)(want < cap ? want : cap);
}
inline bool on16(const void* p) { return ((uintptr_t)p & 15) == 0; }

}  // namespace

IK_EXPORT int ik_dynamic_tanh(const float* x, const int* rows_in, const float* w, const float* b, float alpha, void* out, int out_dtype,
                              int rows, int d, cudaStream_t stream) {
    if (rows < 0 || d <= 0 || !w || !b) return IK_BAD_ARGUMENT;
    if (rows == 0) return IK_OK;
    if ((size_t)rows * d >= 1u << 31) return IK_UNSUPPORTED;
    const unsigned total = (unsigned)rows * d;
    const Dyt n{w, b, alpha};
    const bool v4 = d % 4 == 0 && on16(x) && on16(w) && on16(b) && on16(out);
#define IK_DYT(TO)                                                                                                                \
    if (v4) IK_RETURN_IF_ERROR(ik_launch((dynamic_tanh_kernel<TO, 4>), blocks_for(total / 4), 256, 0, stream, x, rows_in, n, (TO*)out, total, d)); \
    else IK_RETURN_IF_ERROR(ik_launch((dynamic_tanh_kernel<TO, 1>), blocks_for(total), 256, 0, stream, x, rows_in, n, (TO*)out, total, d))
    if (out_dtype == IK_F32) { IK_DYT(float); }
    else if (out_dtype == IK_BF16) { IK_DYT(__nv_bfloat16); }
    else return IK_BAD_ARGUMENT;
#undef IK_DYT
    IK_LAUNCH_STATUS();
}

IK_EXPORT int ik_dynamic_tanh_embed(const int* ids, const void* table, int table_dtype, const float* w, const float* b, float alpha, float* out,
                                    int T, int d, int V, float scale, int* status, cudaStream_t stream) {
    if (T < 0 || d <= 0 || V <= 0 || !w || !b) return IK_BAD_ARGUMENT;
    if (T == 0) return IK_OK;
    if ((size_t)T * d >= 1u << 31) return IK_UNSUPPORTED;
    const unsigned total = (unsigned)T * d;
    const Dyt n{w, b, alpha};
    const bool v4 = d % 4 == 0 && on16(table) && on16(w) && on16(b) && on16(out);
#define IK_DYT_EMBED(TW)                                                                                                                        \
    if (v4) IK_RETURN_IF_ERROR(ik_launch((dynamic_tanh_embed_kernel<TW, 4>), blocks_for(total / 4), 256, 0, stream, ids, (const TW*)table, n, out, total, d, V, scale, status)); \
    else IK_RETURN_IF_ERROR(ik_launch((dynamic_tanh_embed_kernel<TW, 1>), blocks_for(total), 256, 0, stream, ids, (const TW*)table, n, out, total, d, V, scale, status))
    if (table_dtype == IK_F32) { IK_DYT_EMBED(float); }
    else if (table_dtype == IK_BF16) { IK_DYT_EMBED(__nv_bfloat16); }
    else return IK_BAD_ARGUMENT;
#undef IK_DYT_EMBED
    IK_LAUNCH_STATUS();
}

// y [T, d], or (parts [rows, d], weight [T, top] or null, row_of [T * top] or null, extra [T, d] or null, extra_weight [T] or null)
// when y is null.  copy (or null) [T, d] with the next norm's nw, nb, nalpha.
IK_EXPORT int ik_dynamic_tanh_add(const float* y, const float* parts, const float* weight, const int* row_of, const float* extra,
                                  const float* extra_weight, int top, const float* w, const float* b, float alpha, float* residual, float mult,
                                  const float* nw, const float* nb, float nalpha, void* copy, int copy_dtype, int T, int d, cudaStream_t stream) {
    if (T < 0 || d <= 0 || !w || !b || !residual || (!y && (!parts || top <= 0)) || (copy && (!nw || !nb))) return IK_BAD_ARGUMENT;
    if (T == 0) return IK_OK;
    if ((size_t)T * d >= 1u << 31) return IK_UNSUPPORTED;
    const unsigned total = (unsigned)T * d;
    const Dyt n{w, b, alpha}, next{nw, nb, nalpha};
    const Parts s{parts, weight, row_of, extra, extra_weight, top};
    const bool v4 = d % 4 == 0 && on16(y) && on16(parts) && on16(extra) && on16(w) && on16(b) && on16(residual) && on16(nw) && on16(nb) && on16(copy);
#define IK_DYT_ADD(TO, V, SUM)                                                                                                     \
    IK_RETURN_IF_ERROR(ik_launch((dynamic_tanh_add_kernel<TO, V, SUM>), blocks_for(total / V), 256, 0, stream, y, s, n, residual, mult, next, (TO*)copy, total, d))
#define IK_DYT_ADD2(TO)                                                                                  \
    if (y) { if (v4) { IK_DYT_ADD(TO, 4, false); } else { IK_DYT_ADD(TO, 1, false); } }                   \
    else { if (v4) { IK_DYT_ADD(TO, 4, true); } else { IK_DYT_ADD(TO, 1, true); } }
    if (copy_dtype == IK_F32) { IK_DYT_ADD2(float) }
    else if (copy_dtype == IK_BF16) { IK_DYT_ADD2(__nv_bfloat16) }
    else return IK_BAD_ARGUMENT;
#undef IK_DYT_ADD2
#undef IK_DYT_ADD
    IK_LAUNCH_STATUS();
}
