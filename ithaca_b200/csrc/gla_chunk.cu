// Gated linear attention for prompts on the tensor cores: S <- diag(a_t) S + k_t v_t^T, o_t = scale S^T q_t, by chunks of 64 tokens.
//
// With a chunk cut into four blocks of 16 tokens, L_i the running sum of log2 a within i's block (token i included; all of this
// per key channel) and T_J block J's total:
//   own     A_ij = sum_d q_i k_j 2^(sum of log2 a over j+1 .. i) for j <= i;            o_i += sum_j A_ij v_j
//   carry   o_i += sum_d q_i 2^(sum over the chunk's tokens up to i) S_before
//   gain    D = sum_j k_j 2^(sum over the chunk's tokens behind j) v_j^T;                S_after = 2^(sum over the chunk) S_before + D
// A's entry of token i of block I and token j of block J is a product of a factor of i and a factor of j, q_i 2^(from a place between
// them to i) . k_j 2^(from j to that place): the middle of the chunk if it lies between I and J, else the beginning of I.  These
// exponents are never positive.  In block I's own columns the place (the beginning of I) lies in front of j, and k_j's exponent is
// -L_j, which grows as the block forgets; up to 2^100 the product of the two factors still is a rounded one of the true term, and a
// block that forgets more forms its own 16 x 16 entries directly.
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
__device__ __forceinline__ void prefetch_l2(const float* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }
// x and y as sums of two bfloat16 numbers each, packed
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
__device__ __forceinline__ void stage_values(const float* __restrict__ p, int ldp, int off, int t0, int n, int dv, bf16* vh, bf16* vl,
                                             int first, int threads) {
    const int q4 = dv / 4, ld = dv + 8;
    #pragma unroll 8
    for (int idx = first; idx < C * q4; idx += threads) {
        const int r = idx / q4, x = (idx - r * q4) * 4;
        const float4 v = r < n ? *reinterpret_cast<const float4*>(p + (size_t)(t0 + r) * ldp + off + x) : make_float4(0.f, 0.f, 0.f, 0.f);
        uint2 h, l;
        split2(v.x, v.y, h.x, l.x);
        split2(v.z, v.w, h.y, l.y);
        *reinterpret_cast<uint2*>(vh + r * ld + x) = h;
        *reinterpret_cast<uint2*>(vl + r * ld + x) = l;
    }
}

// 16 tokens of two key channels: columns of a matrix with row stride ld, from token t0 on, zeros from token n on.
__device__ __forceinline__ void load16(float2 (&x)[SUB], const float* __restrict__ src, size_t ld, int n) {
    #pragma unroll
    for (int i = 0; i < SUB; i++) x[i] = i < n ? *reinterpret_cast<const float2*>(src + i * ld) : make_float2(0.f, 0.f);
}
__device__ __forceinline__ void running_sums(float2 (&x)[SUB]) {
    #pragma unroll
    for (int i = 1; i < SUB; i++) { x[i].x += x[i - 1].x; x[i].y += x[i - 1].y; }
}
// rows[i] = x_i 2^(base + sign L_i), as two terms, channels d and d + 1 packed; the exponent at most `top`
__device__ __forceinline__ void put16(const float2 (&x)[SUB], const float2 (&L)[SUB], float2 base, float sign, float top, bf16* hi, bf16* lo, int ld) {
    #pragma unroll
    for (int i = 0; i < SUB; i++) {
        uint32_t h, l;
        split2(x[i].x * ex2(fminf(fmaf(sign, L[i].x, base.x), top)), x[i].y * ex2(fminf(fmaf(sign, L[i].y, base.y), top)), h, l);
        *reinterpret_cast<uint32_t*>(hi + i * ld) = h;
        *reinterpret_cast<uint32_t*>(lo + i * ld) = l;
    }
}
__device__ __forceinline__ float2 add2(float2 a, float2 b) { return make_float2(a.x + b.x, a.y + b.y); }

// ------------------------------------------------------------------ gains
// ws[place][h][dv][dk] = D (values x key channels), keep[place][h][dk] = the chunk's decay.  The first 128 threads bring the values,
// the others a block's tokens of two key channels each (IT times).  NK: key channels in eights (at most).
template <int DK, int DV, int IT, int NK>
__global__ void __launch_bounds__(256)
gla_gain_kernel(const float* __restrict__ p, int ldp, int k_off, int v_off, const float* __restrict__ g, const int* __restrict__ cu, int B,
                float* __restrict__ ws, float* __restrict__ keep, int H, int dk_, int dv_) {
    extern __shared__ __align__(16) unsigned char smem[];
    ik_pdl_wait();
    IK_AFTER_WAIT(p);
    IK_AFTER_WAIT(g);
    IK_AFTER_WAIT(cu);
    ik_pdl_launch_dependents();
    int b, c;
    if (!find_chunk(cu, B, blockIdx.x, b, c)) return;
    const int dk = DK ? DK : dk_, dv = DV ? DV : dv_;
    const int h = blockIdx.y, t0 = cu[b] + c * C, n = min(C, cu[b + 1] - t0), ldk = dk + 8, ldv = dv + 8, pairs = dk / 2;
    float* tot = (float*)smem;                              // [NSUB][dk]
    bf16* kh = (bf16*)(tot + NSUB * dk);                    // [C][ldk]
    bf16* kl = kh + C * ldk;
    bf16* vh = kl + C * ldk;                                // [C][ldv]
    bf16* vl = vh + C * ldv;
    const size_t place = (size_t)blockIdx.x * H + h;
    const int mine = (int)threadIdx.x - 128;
    float2 L[IT][SUB], k[IT][SUB];
    if (mine >= 0) {
        #pragma unroll
        for (int it = 0; it < IT; it++) {
            const int item = mine + it * 128, J = item / pairs, d = 2 * (item - J * pairs);
            if (J >= NSUB) break;
            load16(L[it], g + ((size_t)(t0 + J * SUB) * H + h) * dk + d, (size_t)H * dk, n - J * SUB);
            load16(k[it], p + (size_t)(t0 + J * SUB) * ldp + k_off + h * dk + d, ldp, n - J * SUB);
            running_sums(L[it]);
            *reinterpret_cast<float2*>(tot + J * dk + d) = L[it][SUB - 1];
        }
    } else {
        stage_values(p, ldp, v_off + h * dv, t0, n, dv, vh, vl, threadIdx.x, 128);
    }
    __syncthreads();
    if (mine >= 0) {
        #pragma unroll
        for (int it = 0; it < IT; it++) {
            const int item = mine + it * 128, J = item / pairs, d = 2 * (item - J * pairs);
            if (J >= NSUB) break;
            float2 rest = L[it][SUB - 1];                   // of block J and the blocks behind it
            #pragma unroll
            for (int m = 1; m < NSUB; m++) if (m > J) rest = add2(rest, *reinterpret_cast<const float2*>(tot + m * dk + d));
            put16(k[it], L[it], rest, -1.f, 0.f, kh + J * SUB * ldk + d, kl + J * SUB * ldk + d, ldk);
            if (J == 0) *reinterpret_cast<float2*>(keep + place * dk + d) = make_float2(ex2(rest.x), ex2(rest.y));
        }
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
// ws[place] goes from a chunk's gain to the state in front of it, every four floats' place taken by their four leading bfloat16 terms
// and then the four second ones.  A thread has four key channels of one value's column.
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
                uint4 two;
                split2(S.x, S.y, two.x, two.z);
                split2(S.z, S.w, two.y, two.w);
                *reinterpret_cast<uint4*>(w + (size_t)(c0 + j) * per) = two;
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
// Rows of the factors.  Of q: a token's 2^(from its block's beginning), block 3's from the middle, blocks 1 .. 3's from the chunk's
// beginning.  Of k: 2^-(from its block's beginning), blocks 0 and 2's up to their end, blocks 0 and 1's up to the middle.
constexpr int Q_OWN = 0, Q_MIDDLE = 64, Q_START = 80, Q_ROWS = 128;
constexpr int K_OWN = 0, K_END = 64, K_MIDDLE = 96, K_ROWS = 128;

// out[t, h, :] = rmsnorm(o) * norm_w * silu(gate) in bfloat16, gate in columns g_off of p.  The first 128 threads bring q, the
// others k, a block's tokens of two channels each (IT times), all of them the values.  A warp has a block of 16 tokens and half
// of the values (NT eights of them at most).  staged: the state passes through shared memory (over the factors of k).
template <int DK, int DV, int IT, int NT>
__global__ void __launch_bounds__(256, NT <= 8 && IT == 1 ? 2 : 1)
gla_out_kernel(const float* __restrict__ p, int ldp, int q_off, int k_off, int v_off, int g_off, const float* __restrict__ g,
               const int* __restrict__ cu, int B, const float* __restrict__ ws, const float* __restrict__ norm_w, float eps, float scale,
               bf16* __restrict__ out, int H, int dk_, int dv_, int staged) {
    extern __shared__ __align__(16) unsigned char smem[];
    ik_pdl_wait();
    IK_AFTER_WAIT(p);
    IK_AFTER_WAIT(g);
    IK_AFTER_WAIT(cu);
    IK_AFTER_WAIT(ws);
    ik_pdl_launch_dependents();
    int b, c;
    if (!find_chunk(cu, B, blockIdx.x, b, c)) return;
    const int dk = DK ? DK : dk_, dv = DV ? DV : dv_;
    const int h = blockIdx.y, t0 = cu[b] + c * C, n = min(C, cu[b + 1] - t0), ldk = dk + 8, ldv = dv + 8, pairs = dk / 2;
    float* tot = (float*)smem;                              // [NSUB][dk]
    float* ss = tot + NSUB * dk;                            // [2][C] the halves' sums of squares
    int* direct = (int*)(ss + 2 * C);                       // [NSUB] the block forms its own entries directly
    bf16* qh = (bf16*)(direct + NSUB);                      // [Q_ROWS][ldk]
    bf16* ql = qh + Q_ROWS * ldk;
    bf16* vh = ql + Q_ROWS * ldk;                           // [C][ldv]
    bf16* vl = vh + C * ldv;
    bf16* kh = vl + C * ldv;                                // [K_ROWS][ldk], later (staged) the state [dv][ldk]
    bf16* kl = kh + K_ROWS * ldk;
    if (threadIdx.x < NSUB) direct[threadIdx.x] = 0;
    // what is read late sets out for the second-level cache now: the gates and the state in front of the chunk
    for (int f = threadIdx.x & 3; f * 32 < dv; f += 4)
        if ((int)threadIdx.x / 4 < n) prefetch_l2(p + (size_t)(t0 + threadIdx.x / 4) * ldp + g_off + h * dv + f * 32);
    for (int f = threadIdx.x; f * 32 < dv * dk; f += 256) prefetch_l2(ws + ((size_t)blockIdx.x * H + h) * dv * dk + f * 32);
    const bool is_q = threadIdx.x < 128;
    const int mine = threadIdx.x & 127;
    float2 L[IT][SUB], x[IT][SUB];
    #pragma unroll
    for (int it = 0; it < IT; it++) {
        const int item = mine + it * 128, J = item / pairs, d = 2 * (item - J * pairs);
        if (J >= NSUB) break;
        load16(L[it], g + ((size_t)(t0 + J * SUB) * H + h) * dk + d, (size_t)H * dk, n - J * SUB);
        load16(x[it], p + (size_t)(t0 + J * SUB) * ldp + (is_q ? q_off : k_off) + h * dk + d, ldp, n - J * SUB);
        running_sums(L[it]);
        if (is_q) *reinterpret_cast<float2*>(tot + J * dk + d) = L[it][SUB - 1];
    }
    stage_values(p, ldp, v_off + h * dv, t0, n, dv, vh, vl, threadIdx.x, 256);
    __syncthreads();
    #pragma unroll
    for (int it = 0; it < IT; it++) {
        const int item = mine + it * 128, J = item / pairs, d = 2 * (item - J * pairs);
        if (J >= NSUB) break;
        const float2 none = make_float2(0.f, 0.f);
        auto total = [&](int m) { return *reinterpret_cast<const float2*>(tot + m * dk + d); };
        auto put = [&](bf16* hi, bf16* lo, int row, float2 base, float sign, float top) {
            put16(x[it], L[it], base, sign, top, hi + row * ldk + d, lo + row * ldk + d, ldk);
        };
        if (is_q) {
            put(qh, ql, Q_OWN + J * SUB, none, 1.f, 0.f);
            if (J == 3) put(qh, ql, Q_MIDDLE, total(2), 1.f, 0.f);
            if (J > 0) {
                float2 front = total(0);
                if (J > 1) front = add2(front, total(1));
                if (J > 2) front = add2(front, total(2));
                put(qh, ql, Q_START + (J - 1) * SUB, front, 1.f, 0.f);
            }
        } else {
            const float2 own = L[it][SUB - 1];
            if (-fminf(own.x, own.y) > LIMIT) direct[J] = 1;
            put(kh, kl, K_OWN + J * SUB, none, -1.f, LIMIT);
            if ((J & 1) == 0) put(kh, kl, K_END + (J >> 1) * SUB, own, -1.f, 0.f);
            if (J < 2) put(kh, kl, K_MIDDLE + J * SUB, J == 0 ? add2(own, total(1)) : own, -1.f, 0.f);
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
    const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_col = (lane >> 4) * 8;
    #pragma unroll
    for (int np = 0; np < NSUB; np++) {
        if (np > I) continue;
        const bool across = I >= 2 && np < 2;
        const int qr = across && I == 3 ? Q_MIDDLE : Q_OWN + I * SUB;
        const int kr = np == I ? K_OWN + np * SUB : across ? K_MIDDLE + np * SUB : K_END + (np >> 1) * SUB;
        const bf16 *qa = qh + (qr + a_row) * ldk + a_col, *ka = kh + (kr + (lane & 7) + (lane >> 4) * 8) * ldk + ((lane >> 3) & 1) * 8;
        #pragma unroll 4
        for (int ks = 0; ks < dk / 16; ks++) {
            uint32_t ah[4], al[4], bh[4], bl[4];
            ldsm4(ah, qa + ks * 16);
            ldsm4(al, qa + ks * 16 + Q_ROWS * ldk);
            ldsm4(bh, ka + ks * 16);
            ldsm4(bl, ka + ks * 16 + K_ROWS * ldk);
            mma(s[2 * np], ah, bh[0], bh[1]);
            mma(s[2 * np + 1], ah, bh[2], bh[3]);
            mma(s[2 * np], ah, bl[0], bl[1]);
            mma(s[2 * np + 1], ah, bl[2], bl[3]);
            mma(s[2 * np], al, bh[0], bh[1]);
            mma(s[2 * np + 1], al, bh[2], bh[3]);
        }
    }
    // the state in front of the chunk: its two terms on their way while the own tokens' products run
    const uint2* Sg = reinterpret_cast<const uint2*>(ws + ((size_t)blockIdx.x * H + h) * dv * dk);      // [dv][dk / 4][leading, second]
    bf16 *Sh = kh, *Sl = kh + dv * ldk;
    if (staged) {
        __syncthreads();                                    // the factors of k have been read
        const int per_row = dk / 2;
        for (int idx = threadIdx.x; idx < dv * per_row; idx += 256) {
            const int r = idx / per_row, f = idx - r * per_row;
            const unsigned dst = (unsigned)__cvta_generic_to_shared((f & 1 ? Sl : Sh) + r * ldk + (f >> 1) * 4);
            asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(dst), "l"(Sg + idx) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    const bool by_hand = direct[I] != 0;
    #pragma unroll
    for (int np = 0; np < NSUB; np++) {
        if (np != I) continue;
        #pragma unroll
        for (int j = 0; j < 2; j++)
            #pragma unroll
            for (int e = 0; e < 4; e++)
                if (j * 8 + 2 * t + (e & 1) > gq + (e >> 1) * 8) s[2 * np + j][e] = 0.f;
    }
    if (by_hand) {                                          // rare: one entry at a time
        float own[8];
        #pragma unroll 1
        for (int e = 0; e < 8; e++) {
            const int i = I * SUB + gq + ((e >> 1) & 1) * 8, jj = I * SUB + (e >> 2) * 8 + 2 * t + (e & 1);
            float v = 0.f;
            if (jj <= i && i < n) {
                const float *qp = p + (size_t)(t0 + i) * ldp + q_off + h * dk, *kp = p + (size_t)(t0 + jj) * ldp + k_off + h * dk;
                for (int d = 0; d < dk; d++) {
                    float sum = 0.f;
                    for (int m = jj + 1; m <= i; m++) sum += g[((size_t)(t0 + m) * H + h) * dk + d];
                    v = fmaf(qp[d] * kp[d], ex2(sum), v);
                }
            }
            #pragma unroll
            for (int f = 0; f < 8; f++) if (f == e) own[f] = v;
        }
        #pragma unroll
        for (int np = 0; np < NSUB; np++)
            if (np == I)
                #pragma unroll
                for (int f = 0; f < 8; f++) s[2 * np + (f >> 2)][f & 3] = own[f];
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
    // what the state in front of the chunk carries
    const bf16* qs = qh + ((I == 0 ? Q_OWN : Q_START + (I - 1) * SUB) + a_row) * ldk + a_col;
    if (staged) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
    }
    #pragma unroll 4
    for (int ks = 0; ks < dk / 16; ks++) {
        uint32_t ah[4], al[4];
        ldsm4(ah, qs + ks * 16);
        ldsm4(al, qs + ks * 16 + Q_ROWS * ldk);
        #pragma unroll
        for (int j = 0; j < NT; j += 2) {
            if (j < nt) {
                uint32_t bh[4], bl[4];
                if (staged) {
                    const int bt = (n0 + j * 8 + (lane & 7) + (lane >> 4) * 8) * ldk + ks * 16 + ((lane >> 3) & 1) * 8;
                    ldsm4(bh, Sh + bt);
                    ldsm4(bl, Sl + bt);
                } else {
                    #pragma unroll
                    for (int f = 0; f < 4; f++) {           // row gq of eight f >> 1, channels 2 t (+ 1) of half f & 1
                        const uint32_t* src = reinterpret_cast<const uint32_t*>(Sg) + (size_t)(n0 + (j + (f >> 1)) * 8 + gq) * dk
                                              + (ks * 4 + (f & 1) * 2 + (t >> 1)) * 4 + (t & 1);
                        bh[f] = src[0];
                        bl[f] = src[2];
                    }
                }
                mma(o[j], ah, bh[0], bh[1]);
                mma(o[j + 1], ah, bh[2], bh[3]);
                mma(o[j], ah, bl[0], bl[1]);
                mma(o[j + 1], ah, bl[2], bl[3]);
                mma(o[j], al, bh[0], bh[1]);
                mma(o[j + 1], al, bh[2], bh[3]);
            }
        }
    }
    // norm over the head's values, gate: the results by whole rows, through the values' place
    if (!staged) __syncthreads();                           // (staged: every warp was done with the values at the last barrier)
    float* rows = (float*)vh;                               // [C][ldv]
    float r0 = 0.f, r1 = 0.f;
    #pragma unroll
    for (int j = 0; j < NT; j++) {
        if (j >= nt) continue;
        #pragma unroll
        for (int e = 0; e < 4; e++) o[j][e] *= scale;
        r0 = fmaf(o[j][0], o[j][0], fmaf(o[j][1], o[j][1], r0));
        r1 = fmaf(o[j][2], o[j][2], fmaf(o[j][3], o[j][3], r1));
        float* dst = rows + (I * SUB + gq) * ldv + n0 + j * 8 + 2 * t;
        *reinterpret_cast<float2*>(dst) = make_float2(o[j][0], o[j][1]);
        *reinterpret_cast<float2*>(dst + 8 * ldv) = make_float2(o[j][2], o[j][3]);
    }
    #pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
        r0 += __shfl_xor_sync(0xffffffffu, r0, x);
        r1 += __shfl_xor_sync(0xffffffffu, r1, x);
    }
    if (t == 0) { ss[half * C + I * SUB + gq] = r0; ss[half * C + I * SUB + gq + 8] = r1; }
    __syncthreads();
    const int q4 = dv / 4;
    #pragma unroll 8
    for (int idx = threadIdx.x; idx < n * q4; idx += 256) {
        const int r = idx / q4, c4 = (idx - r * q4) * 4;
        const float4 gt = *reinterpret_cast<const float4*>(p + (size_t)(t0 + r) * ldp + g_off + h * dv + c4);
        const float4 w = *reinterpret_cast<const float4*>(norm_w + c4), y = *reinterpret_cast<const float4*>(rows + r * ldv + c4);
        const float inv = rsqrtf((ss[r] + ss[C + r]) / (float)dv + eps);
        auto gated = [&](float a, float v, float wv) { return __fdividef(a, 1.0f + __expf(-a)) * (v * inv * wv); };
        ik_st4(out, ((size_t)(t0 + r) * H + h) * dv + c4, make_float4(gated(gt.x, y.x, w.x), gated(gt.y, y.y, w.y), gated(gt.z, y.z, w.z), gated(gt.w, y.w, w.w)));
    }
}

size_t gain_smem(int dk, int dv) { return (size_t)NSUB * dk * 4 + (size_t)2 * C * (dk + 8 + dv + 8) * 2; }
size_t out_smem(int dk, int dv, bool staged) {
    const size_t rows = staged && dv > K_ROWS ? dv : K_ROWS;
    return (size_t)NSUB * dk * 4 + 2 * C * 4 + NSUB * 4 + (size_t)(2 * (Q_ROWS + rows) * (dk + 8) + 2 * C * (dv + 8)) * 2;
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
    if (dk % 16 || dk > 128 || dv % 32 || dv > 256 || ldp % 4 || q_off % 4 || k_off % 4 || v_off % 4 || g_off % 4 || ((uintptr_t)p & 15) || ((uintptr_t)g & 15) ||
        ((uintptr_t)ws & 15) || ((uintptr_t)keep & 15) || ((uintptr_t)state & 15) || ((uintptr_t)norm_w & 15) || (long long)H * dk * dv > 0x7fffffff ||
        B > 65535 || H > 65535)
        return IK_UNSUPPORTED;
    if (T == 0 || B == 0) return IK_OK;
    const bool staged = out_smem(dk, dv, true) <= 227 * 1024;
    const size_t sg = gain_smem(dk, dv), so = out_smem(dk, dv, staged);
    if (so > 227 * 1024) return IK_UNSUPPORTED;
    const dim3 grid(ik_gla_places(T, B), H);
#define IK_GLA(SMEM, KERN, ...)                                                                                    \
    {                                                                                                              \
        auto kern = KERN;                                                                                          \
        if (SMEM > 48 * 1024) {                                                                                    \
            cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);    \
            if (e != cudaSuccess) return (int)e;                                                                   \
        }                                                                                                          \
        IK_RETURN_IF_ERROR(ik_launch(kern, grid, 256, SMEM, stream, __VA_ARGS__));                                 \
    }
#define IK_GLA_GAIN(DK, DV, IT, NK) IK_GLA(sg, (gla_gain_kernel<DK, DV, IT, NK>), p, ldp, k_off, v_off, g, cu, B, ws, keep, H, dk, dv)
#define IK_GLA_OUT(DK, DV, IT, NT)                                                                                                  \
    IK_GLA(so, (gla_out_kernel<DK, DV, IT, NT>), p, ldp, q_off, k_off, v_off, g_off, g, cu, B, (const float*)ws, norm_w, eps, scale, \
           (bf16*)out, H, dk, dv, staged ? 1 : 0)
    if (dk == 64 && dv == 128) IK_GLA_GAIN(64, 128, 1, 8)
    else if (dk <= 64) IK_GLA_GAIN(0, 0, 1, 8)
    else IK_GLA_GAIN(0, 0, 2, 16)
    IK_RETURN_IF_ERROR(ik_launch(gla_state_kernel, dim3((H * dk * dv / 4 + 127) / 128, B), 128, 0, stream, ws, (const float*)keep, state, slots, cu, kv_lens, H, dk, dv));
    if (dk == 64 && dv == 128) IK_GLA_OUT(64, 128, 1, 8)
    else if (dk <= 64 && dv <= 128) IK_GLA_OUT(0, 0, 1, 8)
    else if (dk <= 64) IK_GLA_OUT(0, 0, 1, 16)
    else if (dv <= 128) IK_GLA_OUT(0, 0, 2, 8)
    else IK_GLA_OUT(0, 0, 2, 16)
#undef IK_GLA_OUT
#undef IK_GLA_GAIN
#undef IK_GLA
    IK_LAUNCH_STATUS();
}
