// Gated linear attention for prompts on the tensor cores: S <- diag(a_t) S + k_t v_t^T, o_t = scale S^T q_t, by chunks of 64 tokens.
//
// With a chunk cut into four blocks of 16 tokens, L_i the running sum of log2 a within i's block (token i included; all of this
// per key channel) and T_J block J's total:
//   own     A_ij = sum_d q_i k_j 2^(sum of log2 a over j+1 .. i) for j <= i;            o_i += sum_j A_ij v_j
//   carry   o_i += sum_d q_i 2^(sum over the chunk's tokens up to i) S_before
//   gain    D = sum_j k_j 2^(sum over the chunk's tokens behind j) v_j^T;                S_after = 2^(sum over the chunk) S_before + D
// No exponent is ever positive but one kind: A's rows of block I are taken as (q_i 2^L_i) . (k_j 2^(rest from j to I's beginning)), the
// rest being a sum of totals and T_J - L_j for J < I, and -L_j for block I's own columns.  The latter grows as the block forgets;
// up to 2^100 a product of the two factors still is a rounded one of the true term, and a block that forgets more forms its own 16 x
// 16 entries directly.
//
// The chunks of all sequences and heads run at once, in three kernels: the gains (D and the chunk's decay), the states in front
// of every chunk (an elementwise recurrence over the chunks, which also takes the sequence's state from its slot and puts
// the new one back), and the outputs with the head's norm and gate as their epilogue.  A float operand is the sum of two
// bfloat16 numbers, a product three products (the low parts' own is left out: relative error near 2^-16), sums are float; the
// state itself and its recurrence are float throughout.
//
// A chunk's place in the workspace is cu[b] / 64 + b + c for chunk c of sequence b: places of different chunks differ, so no
// sequence needs to know how many chunks the ones before it have.
#include <math.h>
#include "common.cuh"

namespace {

typedef __nv_bfloat16 bf16;
constexpr int C = 64, SUB = 16, NSUB = C / SUB;
constexpr float LIMIT = 100.f;                              // the largest exponent of block I's own columns

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
    const uint32_t s = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const void* p) {
    const uint32_t s = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
// x as the sum of two bfloat16 numbers; two x at a time, packed
__device__ __forceinline__ void split(float x, bf16& hi, bf16& lo) { hi = __float2bfloat16_rn(x); lo = __float2bfloat16_rn(x - __bfloat162float(hi)); }
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// The sequence and chunk of workspace place `place`; false where there is none.
__device__ __forceinline__ bool find_chunk(const int* __restrict__ cu, int B, int place, int& b, int& c) {
    int lo = 0, hi = B - 1;                                 // the last sequence whose first place is not behind `place`
    while (lo < hi) {
        const int m = (lo + hi + 1) >> 1;
        if (cu[m] / C + m <= place) lo = m; else hi = m - 1;
    }
    b = lo;
    c = place - (cu[b] / C + b);
    return c >= 0 && c * C < cu[b + 1] - cu[b];
}

// v of the chunk's tokens (zeros behind the last), as two terms: [C][dv + 8] each
__device__ __forceinline__ void stage_values(const float* __restrict__ p, int ldp, int off, int t0, int n, int dv, bf16* vh, bf16* vl) {
    const int q4 = dv / 4, ld = dv + 8;
    #pragma unroll 4
    for (int idx = threadIdx.x; idx < C * q4; idx += 256) {
        const int r = idx / q4, x = (idx - r * q4) * 4;
        const float4 v = r < n ? *reinterpret_cast<const float4*>(p + (size_t)(t0 + r) * ldp + off + x) : make_float4(0.f, 0.f, 0.f, 0.f);
        uint2 h, l;
        split2(v.x, v.y, h.x, l.x);
        split2(v.z, v.w, h.y, l.y);
        *reinterpret_cast<uint2*>(vh + r * ld + x) = h;
        *reinterpret_cast<uint2*>(vl + r * ld + x) = l;
    }
}

// ------------------------------------------------------------------ gains
// ws[place][h][dv][dk] = D (values x key channels), keep[place][h][dk] = the chunk's decay.  IT: (channel, block) pairs a thread
// has, NK: key channels in eights (at most).
template <int IT, int NK>
__global__ void __launch_bounds__(256)
gla_gain_kernel(const float* __restrict__ p, int ldp, int k_off, int v_off, const float* __restrict__ g, const int* __restrict__ cu, int B,
                float* __restrict__ ws, float* __restrict__ keep, int H, int dk, int dv) {
    extern __shared__ __align__(16) unsigned char smem[];
    ik_pdl_wait();
    IK_AFTER_WAIT(p);
    IK_AFTER_WAIT(g);
    IK_AFTER_WAIT(cu);
    ik_pdl_launch_dependents();
    int b, c;
    if (!find_chunk(cu, B, blockIdx.x, b, c)) return;
    const int h = blockIdx.y, t0 = cu[b] + c * C, n = min(C, cu[b + 1] - t0), ldk = dk + 8, ldv = dv + 8;
    float* tot = (float*)smem;                              // [NSUB][dk]
    bf16* kh = (bf16*)(tot + NSUB * dk);                    // [C][ldk]
    bf16* kl = kh + C * ldk;
    bf16* vh = kl + C * ldk;                                // [C][ldv]
    bf16* vl = vh + C * ldv;
    float L[IT][SUB], k[IT][SUB];
    #pragma unroll
    for (int it = 0; it < IT; it++) {
        const int item = threadIdx.x + it * 256, J = item / dk, d = item - J * dk;
        if (J >= NSUB) break;
        #pragma unroll
        for (int i = 0; i < SUB; i++) {
            const int r = J * SUB + i;
            L[it][i] = r < n ? g[((size_t)(t0 + r) * H + h) * dk + d] : 0.f;
            k[it][i] = r < n ? p[(size_t)(t0 + r) * ldp + k_off + h * dk + d] : 0.f;
        }
        #pragma unroll
        for (int i = 1; i < SUB; i++) L[it][i] += L[it][i - 1];
        tot[J * dk + d] = L[it][SUB - 1];
    }
    stage_values(p, ldp, v_off + h * dv, t0, n, dv, vh, vl);
    __syncthreads();
    const size_t place = (size_t)blockIdx.x * H + h;
    #pragma unroll
    for (int it = 0; it < IT; it++) {
        const int item = threadIdx.x + it * 256, J = item / dk, d = item - J * dk;
        if (J >= NSUB) break;
        float behind = 0.f;                                 // of the blocks behind J
        #pragma unroll
        for (int m = NSUB - 1; m >= 0; m--) if (m > J) behind += tot[m * dk + d];
        #pragma unroll
        for (int i = 0; i < SUB; i++) split(k[it][i] * ex2(behind + (L[it][SUB - 1] - L[it][i])), kh[(J * SUB + i) * ldk + d], kl[(J * SUB + i) * ldk + d]);
        if (J == 0) keep[place * dk + d] = ex2(behind + L[it][SUB - 1]);
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, t = lane & 3;
    for (int m0 = warp * 16; m0 < dv; m0 += 128) {
        float acc[NK][4];
        #pragma unroll
        for (int j = 0; j < NK; j++)
            #pragma unroll
            for (int e = 0; e < 4; e++) acc[j][e] = 0.f;
        #pragma unroll
        for (int ks = 0; ks < C / 16; ks++) {
            uint32_t ah[4], al[4];
            const int at = (ks * 16 + (lane & 7) + (lane >> 4) * 8) * ldv + m0 + ((lane >> 3) & 1) * 8;
            ldsm4t(ah, vh + at);
            ldsm4t(al, vl + at);
            #pragma unroll
            for (int j = 0; j < NK; j += 2) {
                if (j * 8 < dk) {
                    uint32_t bh[4], bl[4];
                    const int bt = (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldk + j * 8 + (lane >> 4) * 8;
                    ldsm4t(bh, kh + bt);
                    ldsm4t(bl, kl + bt);
                    mma(acc[j], ah, bh[0], bh[1]);
                    mma(acc[j + 1], ah, bh[2], bh[3]);
                    mma(acc[j], ah, bl[0], bl[1]);
                    mma(acc[j + 1], ah, bl[2], bl[3]);
                    mma(acc[j], al, bh[0], bh[1]);
                    mma(acc[j + 1], al, bh[2], bh[3]);
                }
            }
        }
        float* out = ws + (place * dv + m0) * dk;
        #pragma unroll
        for (int j = 0; j < NK; j++) {
            if (j * 8 >= dk) continue;
            *reinterpret_cast<float2*>(out + (size_t)gq * dk + j * 8 + 2 * t) = make_float2(acc[j][0], acc[j][1]);
            *reinterpret_cast<float2*>(out + (size_t)(gq + 8) * dk + j * 8 + 2 * t) = make_float2(acc[j][2], acc[j][3]);
        }
    }
}

// ------------------------------------------------------------------ states
// ws[place] goes from a chunk's gain to the state in front of it.  A thread has four key channels of one value's column.
__global__ void __launch_bounds__(128)
gla_state_kernel(float* __restrict__ ws, const float* __restrict__ keep, float* __restrict__ state, const int* __restrict__ slots,
                 const int* __restrict__ cu, const int* __restrict__ kv_lens, int H, int dk, int dv) {
    ik_pdl_wait();
    IK_AFTER_WAIT(ws);
    IK_AFTER_WAIT(keep);
    IK_AFTER_WAIT(slots);
    IK_AFTER_WAIT(cu);
    IK_AFTER_WAIT(kv_lens);
    ik_pdl_launch_dependents();
    const int b = blockIdx.y, lo = cu[b], hi = cu[b + 1], end = kv_lens[b], start = end - (hi - lo);
    const int per = H * dk * dv, e = (blockIdx.x * 128 + threadIdx.x) * 4;
    if (e >= per || hi <= lo) return;
    const int h = e / (dk * dv), d = e % dk, n = (hi - lo + C - 1) / C;
    float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
    if (start > 0) S = *reinterpret_cast<const float4*>(state + ((size_t)slots[b] * 2 + ((start - 1) & 1)) * per + e);
    float* w = ws + (size_t)(lo / C + b) * per + e;
    const float* kp = keep + ((size_t)(lo / C + b) * H + h) * dk + d;
    constexpr int AHEAD = 8;
    for (int c0 = 0; c0 < n; c0 += AHEAD) {
        float4 D[AHEAD], K[AHEAD];
        #pragma unroll
        for (int j = 0; j < AHEAD; j++) {
            if (c0 + j < n) {
                D[j] = *reinterpret_cast<const float4*>(w + (size_t)(c0 + j) * per);
                K[j] = *reinterpret_cast<const float4*>(kp + (size_t)(c0 + j) * H * dk);
            }
        }
        #pragma unroll
        for (int j = 0; j < AHEAD; j++) {
            if (c0 + j < n) {
                *reinterpret_cast<float4*>(w + (size_t)(c0 + j) * per) = S;
                S.x = fmaf(K[j].x, S.x, D[j].x);
                S.y = fmaf(K[j].y, S.y, D[j].y);
                S.z = fmaf(K[j].z, S.z, D[j].z);
                S.w = fmaf(K[j].w, S.w, D[j].w);
            }
        }
    }
    *reinterpret_cast<float4*>(state + ((size_t)slots[b] * 2 + ((end - 1) & 1)) * per + e) = S;
}

// ------------------------------------------------------------------ outputs
// out[t, h, :] = rmsnorm(o) * norm_w * silu(gate) in bfloat16, gate in columns g_off of p.  A warp has a block of 16 tokens and
// half of the values (NT eights of them at most).
template <int IT, int NT>
__global__ void __launch_bounds__(256)
gla_out_kernel(const float* __restrict__ p, int ldp, int q_off, int k_off, int v_off, int g_off, const float* __restrict__ g,
               const int* __restrict__ cu, int B, const float* __restrict__ ws, const float* __restrict__ norm_w, float eps, float scale,
               bf16* __restrict__ out, int H, int dk, int dv) {
    extern __shared__ __align__(16) unsigned char smem[];
    ik_pdl_wait();
    IK_AFTER_WAIT(p);
    IK_AFTER_WAIT(g);
    IK_AFTER_WAIT(cu);
    IK_AFTER_WAIT(ws);
    ik_pdl_launch_dependents();
    int b, c;
    if (!find_chunk(cu, B, blockIdx.x, b, c)) return;
    const int h = blockIdx.y, t0 = cu[b] + c * C, n = min(C, cu[b + 1] - t0), ldk = dk + 8, ldv = dv + 8;
    float* tot = (float*)smem;                              // [NSUB][dk]
    float* before = tot + NSUB * dk;                        // [NSUB][dk] 2^(sum over the chunk's tokens in front of the block)
    float* Ls = before + NSUB * dk;                         // [C][dk]
    float* ss = Ls + C * dk;                                // [2][C] the halves' sums of squares
    int* direct = (int*)(ss + 2 * C);                       // [NSUB] the block forms its own entries directly
    bf16* qh = (bf16*)(direct + NSUB);                      // [C][ldk] q 2^L
    bf16* ql = qh + C * ldk;
    bf16* kh = ql + C * ldk;                                // [160][ldk] for blocks 0 .. 3: rows of 16, 32, 48, 64 keys
    bf16* kl = kh + 160 * ldk;
    bf16* vh = kl + 160 * ldk;                              // [C][ldv]
    bf16* vl = vh + C * ldv;
    if (threadIdx.x < NSUB) direct[threadIdx.x] = 0;
    float L[IT][SUB], q[IT][SUB], k[IT][SUB];
    #pragma unroll
    for (int it = 0; it < IT; it++) {
        const int item = threadIdx.x + it * 256, J = item / dk, d = item - J * dk;
        if (J >= NSUB) break;
        #pragma unroll
        for (int i = 0; i < SUB; i++) {
            const int r = J * SUB + i;
            L[it][i] = r < n ? g[((size_t)(t0 + r) * H + h) * dk + d] : 0.f;
            q[it][i] = r < n ? p[(size_t)(t0 + r) * ldp + q_off + h * dk + d] : 0.f;
            k[it][i] = r < n ? p[(size_t)(t0 + r) * ldp + k_off + h * dk + d] : 0.f;
        }
        #pragma unroll
        for (int i = 1; i < SUB; i++) L[it][i] += L[it][i - 1];
        #pragma unroll
        for (int i = 0; i < SUB; i++) Ls[(J * SUB + i) * dk + d] = L[it][i];
        tot[J * dk + d] = L[it][SUB - 1];
    }
    stage_values(p, ldp, v_off + h * dv, t0, n, dv, vh, vl);
    __syncthreads();
    #pragma unroll
    for (int it = 0; it < IT; it++) {
        const int item = threadIdx.x + it * 256, J = item / dk, d = item - J * dk;
        if (J >= NSUB) break;
        float front = 0.f;
        #pragma unroll
        for (int m = 0; m < NSUB; m++) if (m < J) front += tot[m * dk + d];
        before[J * dk + d] = ex2(front);
        if (-L[it][SUB - 1] > LIMIT) direct[J] = 1;
        #pragma unroll
        for (int i = 0; i < SUB; i++) {
            split(q[it][i] * ex2(L[it][i]), qh[(J * SUB + i) * ldk + d], ql[(J * SUB + i) * ldk + d]);
            const int r = 8 * J * (J + 1) + J * SUB + i;    // in block J's own rows, which begin at 8 J (J + 1)
            split(k[it][i] * ex2(fminf(-L[it][i], LIMIT)), kh[r * ldk + d], kl[r * ldk + d]);
        }
        float rest = L[it][SUB - 1];
        #pragma unroll
        for (int I = 1; I < NSUB; I++) {
            if (I <= J) continue;
            #pragma unroll
            for (int i = 0; i < SUB; i++) {
                const int r = 8 * I * (I + 1) + J * SUB + i;
                split(k[it][i] * ex2(rest - L[it][i]), kh[r * ldk + d], kl[r * ldk + d]);
            }
            rest += tot[I * dk + d];
        }
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, t = lane & 3;
    const int half = warp >> 2, I = half ? 7 - warp : warp;              // a scheduler's two warps have one long and one short row
    float s[2 * NSUB][4];
    #pragma unroll
    for (int j = 0; j < 2 * NSUB; j++)
        #pragma unroll
        for (int e = 0; e < 4; e++) s[j][e] = 0.f;
    const bf16 *kbh = kh + 8 * I * (I + 1) * ldk, *kbl = kl + 8 * I * (I + 1) * ldk;
    const int a_at = (I * SUB + (lane & 7) + ((lane >> 3) & 1) * 8) * ldk + (lane >> 4) * 8;
    for (int ks = 0; ks < dk / 16; ks++) {
        uint32_t ah[4], al[4];
        ldsm4(ah, qh + a_at + ks * 16);
        ldsm4(al, ql + a_at + ks * 16);
        #pragma unroll
        for (int np = 0; np < NSUB; np++) {
            if (np <= I) {
                uint32_t bh[4], bl[4];
                const int bt = (np * 16 + (lane & 7) + (lane >> 4) * 8) * ldk + ks * 16 + ((lane >> 3) & 1) * 8;
                ldsm4(bh, kbh + bt);
                ldsm4(bl, kbl + bt);
                mma(s[2 * np], ah, bh[0], bh[1]);
                mma(s[2 * np + 1], ah, bh[2], bh[3]);
                mma(s[2 * np], ah, bl[0], bl[1]);
                mma(s[2 * np + 1], ah, bl[2], bl[3]);
                mma(s[2 * np], al, bh[0], bh[1]);
                mma(s[2 * np + 1], al, bh[2], bh[3]);
            }
        }
    }
    const bool by_hand = direct[I] != 0;
    #pragma unroll
    for (int np = 0; np < NSUB; np++) {
        if (np != I) continue;
        #pragma unroll
        for (int j = 0; j < 2; j++)
            #pragma unroll
            for (int e = 0; e < 4; e++) {
                const int i = gq + (e >> 1) * 8, jj = j * 8 + 2 * t + (e & 1);
                if (jj > i) { s[2 * np + j][e] = 0.f; continue; }
                if (!by_hand) continue;
                float v = 0.f;
                const int ri = I * SUB + i, rj = I * SUB + jj;
                if (ri < n) {
                    const float *qp = p + (size_t)(t0 + ri) * ldp + q_off + h * dk, *kp = p + (size_t)(t0 + rj) * ldp + k_off + h * dk;
                    for (int d = 0; d < dk; d++) v = fmaf(qp[d] * kp[d], ex2(Ls[ri * dk + d] - Ls[rj * dk + d]), v);
                }
                s[2 * np + j][e] = v;
            }
    }
    // own tokens
    const int nt = dv / 16, n0 = half * nt * 8;             // this warp's eights of values, the first value
    float o[NT][4];
    #pragma unroll
    for (int j = 0; j < NT; j++)
        #pragma unroll
        for (int e = 0; e < 4; e++) o[j][e] = 0.f;
    #pragma unroll
    for (int kk = 0; kk < NSUB; kk++) {
        if (kk > I) continue;
        uint32_t ph[4], pl[4];
        split2(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]);
        split2(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
        split2(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]);
        split2(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
        #pragma unroll
        for (int j = 0; j < NT; j += 2) {
            if (j < nt) {
                uint32_t bh[4], bl[4];
                const int bt = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + n0 + j * 8 + (lane >> 4) * 8;
                ldsm4t(bh, vh + bt);
                ldsm4t(bl, vl + bt);
                mma(o[j], ph, bh[0], bh[1]);
                mma(o[j + 1], ph, bh[2], bh[3]);
                mma(o[j], ph, bl[0], bl[1]);
                mma(o[j + 1], ph, bl[2], bl[3]);
                mma(o[j], pl, bh[0], bh[1]);
                mma(o[j + 1], pl, bh[2], bh[3]);
            }
        }
    }
    // what the state in front of the chunk carries, its rows decayed up to the block
    const float* St = ws + (((size_t)blockIdx.x * H + h) * dv + n0 + gq) * dk + 2 * t;
    for (int ks = 0; ks < dk / 16; ks++) {
        uint32_t ah[4], al[4];
        ldsm4(ah, qh + a_at + ks * 16);
        ldsm4(al, ql + a_at + ks * 16);
        const float2 f0 = *reinterpret_cast<const float2*>(before + I * dk + ks * 16 + 2 * t);
        const float2 f1 = *reinterpret_cast<const float2*>(before + I * dk + ks * 16 + 2 * t + 8);
        #pragma unroll
        for (int j = 0; j < NT; j++) {
            if (j < nt) {
                const float2 s0 = *reinterpret_cast<const float2*>(St + (size_t)j * 8 * dk + ks * 16);
                const float2 s1 = *reinterpret_cast<const float2*>(St + (size_t)j * 8 * dk + ks * 16 + 8);
                uint32_t b0h, b0l, b1h, b1l;
                split2(s0.x * f0.x, s0.y * f0.y, b0h, b0l);
                split2(s1.x * f1.x, s1.y * f1.y, b1h, b1l);
                mma(o[j], ah, b0h, b1h);
                mma(o[j], ah, b0l, b1l);
                mma(o[j], al, b0h, b1h);
            }
        }
    }
    // norm over the head's values, gate
    float r0 = 0.f, r1 = 0.f;
    #pragma unroll
    for (int j = 0; j < NT; j++) {
        #pragma unroll
        for (int e = 0; e < 4; e++) o[j][e] *= scale;
        r0 = fmaf(o[j][0], o[j][0], fmaf(o[j][1], o[j][1], r0));
        r1 = fmaf(o[j][2], o[j][2], fmaf(o[j][3], o[j][3], r1));
    }
    #pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
        r0 += __shfl_xor_sync(0xffffffffu, r0, x);
        r1 += __shfl_xor_sync(0xffffffffu, r1, x);
    }
    if (t == 0) { ss[half * C + I * SUB + gq] = r0; ss[half * C + I * SUB + gq + 8] = r1; }
    __syncthreads();
    #pragma unroll
    for (int x = 0; x < 2; x++) {
        const int r = I * SUB + gq + 8 * x;
        if (r >= n) continue;
        const float inv = 1.0f / sqrtf((ss[r] + ss[C + r]) / (float)dv + eps);
        const float* gp = p + (size_t)(t0 + r) * ldp + g_off + h * dv + n0 + 2 * t;
        bf16* op = out + ((size_t)(t0 + r) * H + h) * dv + n0 + 2 * t;
        #pragma unroll
        for (int j = 0; j < NT; j++) {
            if (j < nt) {
                const float2 gt = *reinterpret_cast<const float2*>(gp + j * 8), w = *reinterpret_cast<const float2*>(norm_w + n0 + 2 * t + j * 8);
                *reinterpret_cast<__nv_bfloat162*>(op + j * 8) = __floats2bfloat162_rn(ik_swiglu_fast(gt.x, o[j][2 * x] * inv * w.x),
                                                                                       ik_swiglu_fast(gt.y, o[j][2 * x + 1] * inv * w.y));
            }
        }
    }
}

size_t gain_smem(int dk, int dv) { return (size_t)NSUB * dk * 4 + (size_t)2 * C * (dk + 8 + dv + 8) * 2; }
size_t out_smem(int dk, int dv) {
    return (size_t)(2 * NSUB + C) * dk * 4 + 2 * C * 4 + NSUB * 4 + (size_t)(2 * (C + 160) * (dk + 8) + 2 * C * (dv + 8)) * 2;
}

}  // namespace

// Places of the workspace for T tokens of B sequences.
IK_EXPORT int ik_gla_places(int T, int B) { return T / C + B; }

// q, k, v, gate: columns of the float matrix p (rows ldp apart); g [T, H * dk]: log2 of the decays; ws [places, H, dv, dk] and keep
// [places, H, dk] floats of the caller's; state [slots, 2, H, dv, dk]; out [T, H * dv] bfloat16.
IK_EXPORT int ik_gla_chunks(const float* p, int ldp, int q_off, int k_off, int v_off, int g_off, const float* g, float* ws, float* keep,
                            float* state, const int* slots, const int* cu, const int* kv_lens, const float* norm_w, float eps, float scale,
                            void* out, int T, int B, int H, int dk, int dv, cudaStream_t stream) {
    if (T < 0 || B < 0 || H <= 0 || dk <= 0 || dv <= 0) return IK_BAD_ARGUMENT;
    if (dk % 16 || dk > 128 || dv % 32 || dv > 256 || ldp % 4 || q_off % 4 || k_off % 4 || v_off % 4 || g_off % 4 || ((uintptr_t)p & 15) || ((uintptr_t)ws & 15) ||
        ((uintptr_t)keep & 15) || ((uintptr_t)state & 15) || ((uintptr_t)norm_w & 7) || (long long)H * dk * dv > 0x7fffffff || B > 65535 || H > 65535)
        return IK_UNSUPPORTED;
    if (T == 0 || B == 0) return IK_OK;
    const size_t sg = gain_smem(dk, dv), so = out_smem(dk, dv);
    if (so > 227 * 1024) return IK_UNSUPPORTED;
    const dim3 grid(ik_gla_places(T, B), H);
    cudaError_t e;
#define IK_GLA(KERN, SMEM, ...)                                                                        \
    {                                                                                                  \
        auto kern = KERN;                                                                              \
        if (SMEM > 48 * 1024) {                                                                        \
            e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);    \
            if (e != cudaSuccess) return (int)e;                                                       \
        }                                                                                              \
        IK_RETURN_IF_ERROR(ik_launch(kern, grid, 256, SMEM, stream, __VA_ARGS__));                     \
    }
    if (dk <= 64) IK_GLA((gla_gain_kernel<1, 8>), sg, p, ldp, k_off, v_off, g, cu, B, ws, keep, H, dk, dv)
    else IK_GLA((gla_gain_kernel<2, 16>), sg, p, ldp, k_off, v_off, g, cu, B, ws, keep, H, dk, dv)
    IK_RETURN_IF_ERROR(ik_launch(gla_state_kernel, dim3((H * dk * dv / 4 + 127) / 128, B), 128, 0, stream, ws, (const float*)keep, state, slots, cu, kv_lens, H, dk, dv));
#define IK_GLA_OUT(IT, NT) IK_GLA((gla_out_kernel<IT, NT>), so, p, ldp, q_off, k_off, v_off, g_off, g, cu, B, (const float*)ws, norm_w, eps, scale, (bf16*)out, H, dk, dv)
    if (dk <= 64) { if (dv <= 64) IK_GLA_OUT(1, 4) else if (dv <= 128) IK_GLA_OUT(1, 8) else IK_GLA_OUT(1, 16) }
    else { if (dv <= 64) IK_GLA_OUT(2, 4) else if (dv <= 128) IK_GLA_OUT(2, 8) else IK_GLA_OUT(2, 16) }
#undef IK_GLA_OUT
#undef IK_GLA
    IK_LAUNCH_STATUS();
}
