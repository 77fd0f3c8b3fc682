// One token per sequence of gated linear attention in one kernel: the decay from its low-rank factor, S <- diag(a) S + k v^T,
// o = scale S^T q, the head's RMS norm and its gate.
//
// A block has one head of one sequence.  Its state [dv][dk] passes through registers once: L lanes (a power of two) share a
// value's column, four key channels a lane and turn; a thread asks for up to AHEAD columns' pieces before it needs the decay,
// whose projection, logarithm and exponential run meanwhile.  The state's two copies alternate by position as everywhere: what
// was read is not overwritten, so a step may run twice.
#include <math.h>
#include "common.cuh"

namespace {

constexpr int THREADS = 256;

// NR: float4 pieces of a column a lane has.  Few blocks (BLOCKS 1): eight columns' pieces on the way per thread; many: four, and
// four blocks an SM (measured at 1,024 and 2,048 blocks of 64 x 128: 1.6 to 1.8 times faster than one block's full depth).
template <int L, int NR, int AHEAD, int BLOCKS>
__global__ void __launch_bounds__(THREADS, BLOCKS)
gla_decode_kernel(const float* __restrict__ p, int ldp, int q_off, int k_off, int v_off, int g_off, int a_off, int rank, const float* __restrict__ a2,
                  const float* __restrict__ a2_bias, float power, float* __restrict__ state, const int* __restrict__ slots,
                  const int* __restrict__ kv_lens, const float* __restrict__ norm_w, float eps, float scale, __nv_bfloat16* __restrict__ out, int H,
                  int dk, int dv) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[32];
    float* ds = sm;                                         // [dk] decays
    float* ks = ds + dk;                                    // [dk]
    float* qs = ks + dk;                                    // [dk]
    float* vs = qs + dk;                                    // [dv]
    float* os = vs + dv;                                    // [dv]
    float* low = os + dv;                                   // [rank]
    ik_pdl_wait();
    IK_AFTER_WAIT(p);
    IK_AFTER_WAIT(slots);
    IK_AFTER_WAIT(kv_lens);
    ik_pdl_launch_dependents();
    const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, part = tid % L, group = tid / L;
    constexpr int COLS = THREADS / L;                       // columns at a time
    const int pos = kv_lens[b] - 1;
    const size_t per = (size_t)H * dk * dv, slot = (size_t)slots[b] * 2;
    const float* s_in = state + (slot + ((pos - 1) & 1)) * per + (size_t)h * dv * dk;
    float* s_out = state + (slot + (pos & 1)) * per + (size_t)h * dv * dk;
    const float* row = p + (size_t)b * ldp;
    float4 S[AHEAD][NR];
    auto ask = [&](int c0) {
        #pragma unroll
        for (int i = 0; i < AHEAD; i++) {
            const int col = c0 + i * COLS + group;
            #pragma unroll
            for (int r = 0; r < NR; r++) {
                const int d = 4 * (part + L * r);
                S[i][r] = (pos > 0 && col < dv && d < dk) ? *reinterpret_cast<const float4*>(s_in + (size_t)col * dk + d) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
        }
    };
    ask(0);
    for (int i = tid; i < rank; i += THREADS) low[i] = row[a_off + i];
    for (int i = tid; i < dk; i += THREADS) { ks[i] = row[k_off + h * dk + i]; qs[i] = row[q_off + h * dk + i]; }
    for (int i = tid; i < dv; i += THREADS) vs[i] = row[v_off + h * dv + i];
    __syncthreads();
    for (int d = tid; d < dk; d += THREADS) {
        const int c = h * dk + d;
        float z = a2_bias[c];
        #pragma unroll 16
        for (int r = 0; r < rank; r++) z = fmaf(a2[(size_t)r * H * dk + c], low[r], z);
        ds[d] = expf(power * ((z < 0.f ? z : 0.f) - log1pf(expf(-fabsf(z)))));
    }
    __syncthreads();
    float4 dec[NR], kk[NR], qq[NR];
    #pragma unroll
    for (int r = 0; r < NR; r++) {
        const int d = 4 * (part + L * r);
        const bool in = d < dk;
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        dec[r] = in ? *reinterpret_cast<const float4*>(ds + d) : zero;
        kk[r] = in ? *reinterpret_cast<const float4*>(ks + d) : zero;
        qq[r] = in ? *reinterpret_cast<const float4*>(qs + d) : zero;
    }
    for (int c0 = 0; c0 < dv; c0 += AHEAD * COLS) {
        if (c0 > 0) ask(c0);
        #pragma unroll
        for (int i = 0; i < AHEAD; i++) {
            const int col = c0 + i * COLS + group;
            const float v = col < dv ? vs[col] : 0.f;
            float o = 0.f;
            #pragma unroll
            for (int r = 0; r < NR; r++) {
                const int d = 4 * (part + L * r);
                float4& s = S[i][r];
                s.x = fmaf(dec[r].x, s.x, kk[r].x * v);
                s.y = fmaf(dec[r].y, s.y, kk[r].y * v);
                s.z = fmaf(dec[r].z, s.z, kk[r].z * v);
                s.w = fmaf(dec[r].w, s.w, kk[r].w * v);
                o = fmaf(s.x, qq[r].x, fmaf(s.y, qq[r].y, fmaf(s.z, qq[r].z, fmaf(s.w, qq[r].w, o))));
                if (col < dv && d < dk) *reinterpret_cast<float4*>(s_out + (size_t)col * dk + d) = s;
            }
            #pragma unroll
            for (int x = 1; x < L; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
            if (part == 0 && col < dv) os[col] = scale * o;
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int i = tid; i < dv; i += THREADS) ss = fmaf(os[i], os[i], ss);
    ss = ik_block_sum<THREADS>(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
    for (int i = tid; i < dv; i += THREADS)
        out[((size_t)b * H + h) * dv + i] = __float2bfloat16_rn(ik_swiglu_fast(row[g_off + h * dv + i], os[i] * inv * norm_w[i]));
}

}  // namespace

// q, k, v, gate and the decay's factor: columns of the float matrix p [B, ..] (rows ldp apart); a2 [rank, H * dk]; state [slots, 2, H, dv,
// dk]; out [B, H * dv] bfloat16.
IK_EXPORT int ik_gla_decode(const float* p, int ldp, int q_off, int k_off, int v_off, int g_off, int a_off, int rank, const float* a2,
                            const float* a2_bias, float power, float* state, const int* slots, const int* kv_lens, const float* norm_w, float eps,
                            float scale, void* out, int B, int H, int dk, int dv, cudaStream_t stream) {
    if (B < 0 || H <= 0 || dk <= 0 || dv <= 0 || rank <= 0 || !a2 || !a2_bias) return IK_BAD_ARGUMENT;
    if (dk % 4 || dk > 512 || B > 65535 || ((uintptr_t)state & 15)) return IK_UNSUPPORTED;
    const size_t smem = (size_t)(3 * dk + 2 * dv + rank) * sizeof(float);
    if (smem > 48 * 1024) return IK_UNSUPPORTED;
    if (B == 0) return IK_OK;
    int L = 1;
    while (L < 32 && 4 * L < dk) L *= 2;
    const bool many = (long long)B * H > 2ll * ik_sm_count();
#define IK_GLA_DEC2(L_, NR_, AHEAD_, BLOCKS_)                                                                                             \
    IK_RETURN_IF_ERROR(ik_launch((gla_decode_kernel<L_, NR_, AHEAD_, BLOCKS_>), dim3(H, B), THREADS, smem, stream, p, ldp, q_off, k_off, v_off, g_off, \
                                 a_off, rank, a2, a2_bias, power, state, slots, kv_lens, norm_w, eps, scale, (__nv_bfloat16*)out, H, dk, dv))
#define IK_GLA_DEC(L_) { if (many) IK_GLA_DEC2(L_, 1, 4, 4); else IK_GLA_DEC2(L_, 1, 8, 1); break; }
    switch (L) {
        case 1: IK_GLA_DEC(1)
        case 2: IK_GLA_DEC(2)
        case 4: IK_GLA_DEC(4)
        case 8: IK_GLA_DEC(8)
        case 16: IK_GLA_DEC(16)
        default:
            if (dk <= 128) IK_GLA_DEC(32)
            else if (dk <= 256) IK_GLA_DEC2(32, 2, 4, 2);
            else IK_GLA_DEC2(32, 4, 4, 1);
    }
#undef IK_GLA_DEC2
#undef IK_GLA_DEC
    IK_LAUNCH_STATUS();
}
