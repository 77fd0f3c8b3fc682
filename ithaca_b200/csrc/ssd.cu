// State-space duality ("mamba2"): a mixer whose state is a matrix per head that decays by one factor per token and head.
//
// Per head h (its B and C come from group h / (H / G)), with x [P], B and C [N], a step dt = softplus(raw + bias) and a rate
// A_h < 0:   S <- exp(A_h dt) S + dt B x^T   (S is N x P, zero before the first token);   y = S^T C + D_h x.
// The mixer's result is y * silu(z), RMS-normed in equal parts of the row, times a weight (gated_group_norm below).
//
// Tokens, slots and positions as everywhere (recurrent.cu): sequence b brings tokens cu_seqlens[b] .. cu_seqlens[b+1] - 1 that
// end at position kv_lens[b] - 1; a sequence whose first token sits at position 0 starts from zeros whatever its slot holds.
// The state lies in slot slots[b] as float [2][H][N][P]: two copies by the parity of the position the state belongs to, so a
// decode step never overwrites what it read and may be run again.
//
// x, B and C are columns of `u`, the output of the short convolution: x from 0, B from H*P, C from H*P + G*N.  The step's raw
// values are columns of `p` (float, row stride ldp) from dt_off.  Steps, decays, states and sums are float.
//
// Three kernels:
//   ssd_scan     one token after the other on the CUDA cores, any sizes; the float32 path's kernel for prompts and single
//                tokens alike (a token gives the same bits however a prompt is cut).
//   ssd_chunk    bfloat16 inputs, prompts: chunks of 64 tokens on the warp-level tensor path (ssd_tcgen05.cu has the form for
//                tcgen05, which takes fewer sizes and is several times faster).
//   ssd_decode   bfloat16 path, one token per sequence: convolution, step, decay, update and read-out in one pass over the
//                state.
#include "common.cuh"

namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float ik_softplusf(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float ik_siluf(float x) { return x / (1.0f + expf(-x)); }

// ------------------------------------------------------------------ token by token
// A block holds 32 columns of one head's S for one sequence: thread (j, part) keeps rows part*R .. part*R + R - 1 of column j
// in registers, one warp per part.  Tokens come through shared memory in tiles (B, C, the block's columns of x, and per token
// the step and the decay); the parts' sums of a column are added in part order.  exact: step and decay are formed in double
// and rounded once (a decay's error is multiplied into the state at every token).
constexpr int SCAN_TT = 16;

template <typename TU, int RMAX>
__global__ void __launch_bounds__(512)
ssd_scan_kernel(const TU* __restrict__ u, int ldu, const float* __restrict__ p, int ldp, int dt_off, const float* __restrict__ dt_bias,
                const float* __restrict__ A, const float* __restrict__ Dv, float* __restrict__ state, const int* __restrict__ slots,
                const int* __restrict__ cu_seqlens, const int* __restrict__ kv_lens, float* __restrict__ out, int H, int G, int N,
                int P, int R, int exact) {
    extern __shared__ __align__(16) float sm[];          // [TT][W]: B, C (N each), x (32), step, decay;  [TT][parts][32] sums
    ik_pdl_wait();
    IK_AFTER_WAIT(u);
    IK_AFTER_WAIT(p);
    IK_AFTER_WAIT(slots);
    IK_AFTER_WAIT(cu_seqlens);
    IK_AFTER_WAIT(kv_lens);
    ik_pdl_launch_dependents();
    const int b = blockIdx.x, h = blockIdx.y, j = threadIdx.x, part = threadIdx.y, parts = blockDim.y;
    const int col0 = blockIdx.z * 32, col = col0 + j;
    const bool live = col < P;
    const int ccol = live ? col : P - 1;
    const int tid = part * 32 + j, nthreads = parts * 32, W = 2 * N + 34;
    float* partial = sm + SCAN_TT * W;
    const int lo = cu_seqlens[b], hi = cu_seqlens[b + 1], end = kv_lens[b], start = end - (hi - lo);
    if (hi <= lo) return;
    const int grp = h / (H / G), b_off = H * P + grp * N, c_off = H * P + G * N + grp * N;
    const size_t per = (size_t)H * N * P;
    const float* st_in = state + ((size_t)slots[b] * 2 + ((start - 1) & 1)) * per + (size_t)h * N * P;
    float* st_out = state + ((size_t)slots[b] * 2 + ((end - 1) & 1)) * per + (size_t)h * N * P;
    const float rate = A[h], bias = dt_bias[h], skip = Dv[h];
    float S[RMAX];
    #pragma unroll
    for (int r = 0; r < RMAX; r++) {
        const int i = part * R + r;
        S[r] = (r < R && i < N && start > 0) ? st_in[(size_t)i * P + ccol] : 0.f;
    }
    for (int t0 = lo; t0 < hi; t0 += SCAN_TT) {
        const int n_here = min(SCAN_TT, hi - t0);
        for (int tt = part; tt < n_here; tt += parts) {
            const TU* row = u + (size_t)(t0 + tt) * ldu;
            float* dst = sm + tt * W;
            for (int w = j; w < N; w += 32) {
                dst[w] = ik_ld(row, b_off + w);
                dst[N + w] = ik_ld(row, c_off + w);
            }
            dst[2 * N + j] = live ? ik_ld(row, h * P + col) : 0.f;
            if (j == 0) {
                const float raw = p[(size_t)(t0 + tt) * ldp + dt_off + h];
                if (exact) {
                    const double z = (double)raw + (double)bias, sp = z > 30.0 ? z : log1p(exp(z));
                    dst[2 * N + 32] = (float)sp;
                    dst[2 * N + 33] = (float)exp((double)rate * sp);
                } else {
                    const float sp = ik_softplusf(raw + bias);
                    dst[2 * N + 32] = sp;
                    dst[2 * N + 33] = expf(rate * sp);
                }
            }
        }
        __syncthreads();
        for (int tt = 0; tt < n_here; tt++) {
            const float* row = sm + tt * W;
            const float* Bn = row + part * R;
            const float* Cn = Bn + N;
            const float a = row[2 * N + 33], xd = row[2 * N + 32] * row[2 * N + j];
            float acc0 = 0.f, acc1 = 0.f;
            #pragma unroll
            for (int r = 0; r < RMAX; r++) {
                if (r < R && part * R + r < N) {
                    S[r] = fmaf(a, S[r], Bn[r] * xd);
                    if (r & 1) acc1 = fmaf(S[r], Cn[r], acc1);
                    else acc0 = fmaf(S[r], Cn[r], acc0);
                }
            }
            partial[(tt * parts + part) * 32 + j] = acc0 + acc1;
        }
        __syncthreads();
        for (int e = tid; e < n_here * 32; e += nthreads) {
            const int tt = e >> 5, jj = e & 31;
            if (col0 + jj >= P) continue;
            float o = 0.f;
            for (int pp = 0; pp < parts; pp++) o += partial[(tt * parts + pp) * 32 + jj];
            out[(size_t)(t0 + tt) * H * P + h * P + col0 + jj] = fmaf(skip, sm[tt * W + 2 * N + jj], o);
        }
        __syncthreads();
    }
    if (live) {
        #pragma unroll
        for (int r = 0; r < RMAX; r++) {
            const int i = part * R + r;
            if (r < R && i < N) st_out[(size_t)i * P + col] = S[r];
        }
    }
}

// ------------------------------------------------------------------ chunks of 64 tokens on the tensor cores
// With c_i the sum of A dt over the chunk's tokens up to and including i (so exp(c_i - c_j) is the decay from j to i):
//   y_i = exp(c_i) S^T C_i + sum_{j <= i} exp(c_i - c_j) dt_j (C_i . B_j) x_j,
//   S  <- exp(c_last) S + sum_j exp(c_last - c_j) dt_j B_j x_j^T.
// A block owns 16 columns of S per warp of one head of one sequence and walks the chunks in order; S^T stays in the
// accumulators of its products (rows: columns p of S, 16 per warp; columns: the N states) and is float throughout.  The
// products take bfloat16 operands: x, B and C are that already; a float operand (the state, the decayed scores, x times its
// weight) is handed over as the sum of two or three bfloat16 numbers, each product with a term of its own, so that its
// relative error is 2^-17 (scores and weighted x) and 2^-25 (state), not 2^-9.  Everything else is float.
//   1. scores (C B^T, rows i dealt to the warps, only j <= i), times decay and step, as two bfloat16 matrices in shared memory;
//   2. y^T = S^T C^T, columns times exp(c_i);   3. y^T += x^T scores^T;   4. S^T <- exp(c_last) S^T + (w x)^T B.
// The next chunk's x, B and C are on their way (cp.async) meanwhile.  Places beyond the sequence's tokens are zeros with a
// step of zero: they leave the state alone.
constexpr int Q = 64;

__device__ __forceinline__ void sd_cp16(void* smem, const void* gmem, bool valid) {
    const uint32_t s = (uint32_t)__cvta_generic_to_shared(smem);
    const int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" :: "r"(s), "l"(gmem), "r"(n));
}
__device__ __forceinline__ void sd_ldsm4(uint32_t (&r)[4], const void* p) {
    const uint32_t s = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void sd_ldsm4t(uint32_t (&r)[4], const void* p) {
    const uint32_t s = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void sd_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two floats as `hi` plus a rest: the pair's leading bfloat16 parts, packed; the floats become what is left of them.
__device__ __forceinline__ uint32_t sd_take(float& a, float& b) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    const uint32_t w = *reinterpret_cast<const uint32_t*>(&v);
    a -= __uint_as_float(w << 16);
    b -= __uint_as_float(w & 0xffff0000u);
    return w;
}
__device__ __forceinline__ float sd_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float sd_hi(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }

template <int NP, int NW>                                  // states padded to NP (a multiple of 16), warps
constexpr size_t ssd_chunk_smem() {
    return (size_t)2 * (2 * Q * (NP + 8) + Q * (16 * NW + 8)) * sizeof(bf16) + (size_t)2 * Q * (Q + 8) * sizeof(bf16) + (size_t)NW * 3 * Q * sizeof(float);
}

template <int NP, int NW>
__global__ void __launch_bounds__(32 * NW)
ssd_chunk_kernel(const bf16* __restrict__ u, int ldu, const float* __restrict__ p, int ldp, int dt_off, const float* __restrict__ dt_bias,
                 const float* __restrict__ A, const float* __restrict__ Dv, float* __restrict__ state, const int* __restrict__ slots,
                 const int* __restrict__ cu_seqlens, const int* __restrict__ kv_lens, float* __restrict__ out, int H, int G, int N, int P) {
    constexpr int PT = 16 * NW, LN = NP + 8, LP = PT + 8, LM = Q + 8, THREADS = 32 * NW, KN = NP / 16;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16* Cs = (bf16*)smem_raw;                            // [2][Q][LN]
    bf16* Bs = Cs + 2 * Q * LN;                            // [2][Q][LN]
    bf16* Xs = Bs + 2 * Q * LN;                            // [2][Q][LP]
    bf16* Mh = Xs + 2 * Q * LP;                            // [Q][LM] decayed scores, leading part: row i, column j
    bf16* Ml = Mh + Q * LM;                                // ... and the rest
    float* cw_all = (float*)(Ml + Q * LM);                 // [NW][3][Q]: c_i in two parts and dt_i, a copy per warp
    ik_pdl_wait();
    IK_AFTER_WAIT(u);
    IK_AFTER_WAIT(p);
    IK_AFTER_WAIT(slots);
    IK_AFTER_WAIT(cu_seqlens);
    IK_AFTER_WAIT(kv_lens);
    ik_pdl_launch_dependents();
    const int h = blockIdx.x, b = blockIdx.y, p0 = blockIdx.z * PT;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int lo = cu_seqlens[b], hi = cu_seqlens[b + 1], end = kv_lens[b], start = end - (hi - lo);
    if (hi <= lo) return;
    const int grp = h / (H / G), x_off = h * P + p0, b_off = H * P + grp * N, c_off = H * P + G * N + grp * N;
    const size_t per = (size_t)H * N * P;
    const float* st_in = state + ((size_t)slots[b] * 2 + ((start - 1) & 1)) * per + (size_t)h * N * P;
    float* st_out = state + ((size_t)slots[b] * 2 + ((end - 1) & 1)) * per + (size_t)h * N * P;
    const float rate = A[h], bias = dt_bias[h], skip = Dv[h];
    float* cw = cw_all + warp * 3 * Q;
    float* cl = cw + Q;
    float* dw = cl + Q;
    // exp(c_i - c_j): c may be large (a token that forgets everything) where the difference is small, so c is kept as the sum of
    // two floats
    auto decay = [&](int i, int j) -> float { return __expf((cw[i] - cw[j]) + (cl[i] - cl[j])); };

    auto load = [&](int t0, int buf) {
        bf16* cs = Cs + buf * Q * LN;
        bf16* bs = Bs + buf * Q * LN;
        bf16* xs = Xs + buf * Q * LP;
        for (int idx = threadIdx.x; idx < Q * (NP / 8); idx += THREADS) {
            const int r = idx / (NP / 8), c = (idx % (NP / 8)) * 8;
            const bool ok = t0 + r < hi && c < N;
            const bf16* row = u + (size_t)(ok ? t0 + r : lo) * ldu;
            sd_cp16(cs + r * LN + c, ok ? row + c_off + c : u, ok);
            sd_cp16(bs + r * LN + c, ok ? row + b_off + c : u, ok);
        }
        for (int idx = threadIdx.x; idx < Q * (PT / 8); idx += THREADS) {
            const int r = idx / (PT / 8), c = (idx % (PT / 8)) * 8;
            const bool ok = t0 + r < hi && p0 + c < P;
            sd_cp16(xs + r * LP + c, ok ? u + (size_t)(t0 + r) * ldu + x_off + c : u, ok);
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    auto raw_step = [&](int t0, int i) -> float { return t0 + i < hi ? p[(size_t)(t0 + i) * ldp + dt_off + h] : 0.f; };

    // S^T: tile n holds states 8n + 2t, + 1 of columns p = g (elements 0, 1) and g + 8 (elements 2, 3) of this warp's sixteen
    const int pa = p0 + warp * 16 + g, pb = pa + 8;
    float S[2 * KN][4];
    #pragma unroll
    for (int n = 0; n < 2 * KN; n++)
        #pragma unroll
        for (int e = 0; e < 4; e++) {
            const int i = n * 8 + 2 * t + (e & 1), pp = e < 2 ? pa : pb;
            S[n][e] = (start > 0 && i < N && pp < P) ? st_in[(size_t)i * P + pp] : 0.f;
        }
    load(lo, 0);
    float raw0 = raw_step(lo, lane), raw1 = raw_step(lo, lane + 32);
    int buf = 0;
    for (int t0 = lo; t0 < hi; t0 += Q, buf ^= 1) {
        // steps and their running sums: every warp for itself, lane l the tokens l and l + 32
        {
            const float d0 = t0 + lane < hi ? ik_softplusf(raw0 + bias) : 0.f, d1 = t0 + lane + 32 < hi ? ik_softplusf(raw1 + bias) : 0.f;
            double s0 = (double)rate * d0, s1 = (double)rate * d1;
            #pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const double q0 = __shfl_up_sync(0xffffffffu, s0, o), q1 = __shfl_up_sync(0xffffffffu, s1, o);
                if (lane >= o) { s0 += q0; s1 += q1; }
            }
            s1 += __shfl_sync(0xffffffffu, s0, 31);
            __syncwarp();
            cw[lane] = (float)s0; cw[lane + 32] = (float)s1;
            cl[lane] = (float)(s0 - (double)(float)s0); cl[lane + 32] = (float)(s1 - (double)(float)s1);
            dw[lane] = d0; dw[lane + 32] = d1;
            __syncwarp();
        }
        asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        __syncthreads();                                   // this chunk is here, and everyone is done with the other buffer and the scores
        if (t0 + Q < hi) {
            load(t0 + Q, buf ^ 1);
            raw0 = raw_step(t0 + Q, lane);
            raw1 = raw_step(t0 + Q, lane + 32);
        }
        const bf16* cs = Cs + buf * Q * LN;
        const bf16* bs = Bs + buf * Q * LN;
        const bf16* xs = Xs + buf * Q * LP;
        // 1. the scores of rows 16 it .. 16 it + 15 with the columns up to there
        #pragma unroll 1
        for (int it = warp; it < Q / 16; it += NW) {
            float sc[Q / 8][4];
            #pragma unroll
            for (int n = 0; n < Q / 8; n++)
                #pragma unroll
                for (int e = 0; e < 4; e++) sc[n][e] = 0.f;
            #pragma unroll
            for (int k = 0; k < KN; k++) {
                uint32_t af[4];
                sd_ldsm4(af, cs + (it * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LN + k * 16 + (lane >> 4) * 8);
                #pragma unroll
                for (int n2 = 0; n2 < Q / 16; n2++) {
                    if (n2 > it) break;
                    uint32_t bfr[4];
                    sd_ldsm4(bfr, bs + (n2 * 16 + (lane & 7) + (lane >> 4) * 8) * LN + k * 16 + ((lane >> 3) & 1) * 8);
                    sd_mma(sc[2 * n2], af, bfr[0], bfr[1]);
                    sd_mma(sc[2 * n2 + 1], af, bfr[2], bfr[3]);
                }
            }
            #pragma unroll
            for (int n = 0; n < Q / 8; n++) {
                if (n > 2 * it + 1) break;
                const int j = n * 8 + 2 * t;
                const float d0 = dw[j], d1 = dw[j + 1];
                #pragma unroll
                for (int r = 0; r < 2; r++) {
                    const int i = it * 16 + g + 8 * r;
                    float m0 = j <= i ? sc[n][2 * r] * (decay(i, j) * d0) : 0.f;
                    float m1 = j + 1 <= i ? sc[n][2 * r + 1] * (decay(i, j + 1) * d1) : 0.f;
                    *reinterpret_cast<uint32_t*>(Mh + i * LM + j) = sd_take(m0, m1);
                    *reinterpret_cast<uint32_t*>(Ml + i * LM + j) = sd_take(m0, m1);
                }
            }
        }
        // 2. what the state carries into the chunk
        float y[Q / 8][4];
        #pragma unroll
        for (int n = 0; n < Q / 8; n++)
            #pragma unroll
            for (int e = 0; e < 4; e++) y[n][e] = 0.f;
        #pragma unroll
        for (int k = 0; k < KN; k++) {
            uint32_t a0[4], a1[4], a2[4];
            #pragma unroll
            for (int e = 0; e < 4; e++) {                  // (row g, k 2t), (row g + 8, k 2t), (row g, k 2t + 8), (row g + 8, k 2t + 8)
                float v0 = S[2 * k + (e >> 1)][2 * (e & 1)], v1 = S[2 * k + (e >> 1)][2 * (e & 1) + 1];
                a0[e] = sd_take(v0, v1);
                a1[e] = sd_take(v0, v1);
                a2[e] = sd_take(v0, v1);
            }
            #pragma unroll
            for (int n2 = 0; n2 < Q / 16; n2++) {
                uint32_t bfr[4];
                sd_ldsm4(bfr, cs + (n2 * 16 + (lane & 7) + (lane >> 4) * 8) * LN + k * 16 + ((lane >> 3) & 1) * 8);
                sd_mma(y[2 * n2], a2, bfr[0], bfr[1]);
                sd_mma(y[2 * n2 + 1], a2, bfr[2], bfr[3]);
                sd_mma(y[2 * n2], a1, bfr[0], bfr[1]);
                sd_mma(y[2 * n2 + 1], a1, bfr[2], bfr[3]);
                sd_mma(y[2 * n2], a0, bfr[0], bfr[1]);
                sd_mma(y[2 * n2 + 1], a0, bfr[2], bfr[3]);
            }
        }
        #pragma unroll
        for (int n = 0; n < Q / 8; n++) {
            const float e0 = __expf(cw[n * 8 + 2 * t]), e1 = __expf(cw[n * 8 + 2 * t + 1]);
            y[n][0] *= e0; y[n][1] *= e1; y[n][2] *= e0; y[n][3] *= e1;
        }
        __syncthreads();                                   // the scores are written
        // 3. the chunk's own tokens, and 4. the state behind them: both read x^T, 16 tokens at a time
        const float keep = __expf(cw[Q - 1]);
        #pragma unroll
        for (int n = 0; n < 2 * KN; n++)
            #pragma unroll
            for (int e = 0; e < 4; e++) S[n][e] *= keep;
        #pragma unroll
        for (int k = 0; k < Q / 16; k++) {
            uint32_t xf[4];
            sd_ldsm4t(xf, xs + (k * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * LP + warp * 16 + ((lane >> 3) & 1) * 8);
            #pragma unroll
            for (int n2 = 0; n2 < Q / 16; n2++) {
                if (n2 < k) continue;                      // columns i of the tile all lie before its rows j
                uint32_t bh[4], bl[4];
                const int at = (n2 * 16 + (lane & 7) + (lane >> 4) * 8) * LM + k * 16 + ((lane >> 3) & 1) * 8;
                sd_ldsm4(bl, Ml + at);
                sd_ldsm4(bh, Mh + at);
                sd_mma(y[2 * n2], xf, bl[0], bl[1]);
                sd_mma(y[2 * n2 + 1], xf, bl[2], bl[3]);
                sd_mma(y[2 * n2], xf, bh[0], bh[1]);
                sd_mma(y[2 * n2 + 1], xf, bh[2], bh[3]);
            }
            uint32_t wh[4], wl[4];
            #pragma unroll
            for (int e = 0; e < 4; e++) {                  // elements e: tokens j = 16 k + 2t, + 1 (e < 2) or + 8, + 9
                const int j = k * 16 + 2 * t + (e >> 1) * 8;
                float v0 = sd_lo(xf[e]) * (decay(Q - 1, j) * dw[j]), v1 = sd_hi(xf[e]) * (decay(Q - 1, j + 1) * dw[j + 1]);
                wh[e] = sd_take(v0, v1);
                wl[e] = sd_take(v0, v1);
            }
            #pragma unroll
            for (int n2 = 0; n2 < KN; n2++) {
                uint32_t bfr[4];
                sd_ldsm4t(bfr, bs + (k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LN + n2 * 16 + (lane >> 4) * 8);
                sd_mma(S[2 * n2], wl, bfr[0], bfr[1]);
                sd_mma(S[2 * n2 + 1], wl, bfr[2], bfr[3]);
                sd_mma(S[2 * n2], wh, bfr[0], bfr[1]);
                sd_mma(S[2 * n2 + 1], wh, bfr[2], bfr[3]);
            }
        }
        #pragma unroll
        for (int n = 0; n < Q / 8; n++)
            #pragma unroll
            for (int e = 0; e < 4; e++) {
                const int i = n * 8 + 2 * t + (e & 1), pp = e < 2 ? pa : pb;
                if (t0 + i < hi && pp < P)
                    out[(size_t)(t0 + i) * H * P + h * P + pp] = fmaf(skip, __bfloat162float(xs[i * LP + pp - p0]), y[n][e]);
            }
    }
    #pragma unroll
    for (int n = 0; n < 2 * KN; n++)
        #pragma unroll
        for (int e = 0; e < 4; e++) {
            const int i = n * 8 + 2 * t + (e & 1), pp = e < 2 ? pa : pb;
            if (i < N && pp < P) st_out[(size_t)i * P + pp] = S[n][e];
        }
}

// ------------------------------------------------------------------ one token per sequence
// Block (head, sequence, up to 64 columns): thread (pv, slice) holds four neighbouring columns of the state's rows slice,
// slice + n_slices, ... .  It asks for them first, then the block forms the convolution of its x, B and C from `p` (the
// projections themselves: x from x_off, then B and C as in `u`, then the raw steps) and the ring of earlier inputs, and then
// the state is advanced, read out and written to the other parity's copy.  Every block convolves its group's B and C for
// itself; the blocks of the group's first head put the new inputs into the ring (at a place that no block reads in this step).
constexpr int DEC_ROWS = 8, DEC_THREADS = 256;              // state rows a thread has in flight

template <int TAPS>                                        // 0: any number, given by `taps_given`
__global__ void __launch_bounds__(DEC_THREADS)
ssd_decode_kernel(const float* __restrict__ p, int ldp, int x_off, const float* __restrict__ cw, const float* __restrict__ cb,
                  float* __restrict__ ring, const float* __restrict__ dt_bias, const float* __restrict__ A, const float* __restrict__ Dv,
                  float* __restrict__ state, const int* __restrict__ slots, const int* __restrict__ cu_seqlens,
                  const int* __restrict__ kv_lens, float* __restrict__ out, int H, int G, int N, int P, int taps_given, int pv_n) {
    extern __shared__ __align__(16) float sm[];            // x [4 pv_n], B [N], C [N], sums [slices][4 pv_n]
    ik_pdl_wait();
    IK_AFTER_WAIT(p);
    IK_AFTER_WAIT(slots);
    IK_AFTER_WAIT(cu_seqlens);
    IK_AFTER_WAIT(kv_lens);
    ik_pdl_launch_dependents();
    const int h = blockIdx.x, b = blockIdx.y, PT = 4 * pv_n, p0 = blockIdx.z * PT;
    const int pv = threadIdx.x % pv_n, slice = threadIdx.x / pv_n, slices = DEC_THREADS / pv_n;
    const int taps = TAPS ? TAPS : taps_given;
    const int tok = cu_seqlens[b], slot = slots[b], end = kv_lens[b], pos = end - 1;
    const int grp = h / (H / G), C_all = H * P + 2 * G * N;
    const size_t per = (size_t)H * N * P;
    const int col = p0 + 4 * pv;
    const bool live = col < P;
    const float* st_in = state + ((size_t)slot * 2 + ((pos - 1) & 1)) * per + (size_t)h * N * P + (live ? col : 0);
    float* st_out = state + ((size_t)slot * 2 + (pos & 1)) * per + (size_t)h * N * P + (live ? col : 0);
    float4 S[DEC_ROWS];
    auto fetch = [&](int n0) {
        #pragma unroll
        for (int r = 0; r < DEC_ROWS; r++) {
            const int n = n0 + slice + r * slices;
            S[r] = (pos > 0 && live && n < N) ? *reinterpret_cast<const float4*>(st_in + (size_t)n * P) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    };
    fetch(0);
    const float* row = p + (size_t)tok * ldp + x_off;      // the convolution's inputs, then the raw steps
    float* rg = ring ? ring + (size_t)slot * taps * C_all : nullptr;
    const bool own_bc = h % (H / G) == 0 && blockIdx.z == 0;
    // channel of the block's e-th convolved value, -1 beyond the head's columns
    auto channel = [&](int e) -> int {
        if (e < PT) return p0 + e < P ? h * P + p0 + e : -1;
        const int w = e - PT;
        return H * P + (w < N ? grp * N + w : G * N + grp * N + w - N);
    };
    const int at = pos % taps;                             // position p of a sequence lies in place p mod taps of its ring
    #pragma unroll 2
    for (int e = threadIdx.x; e < PT + 2 * N; e += DEC_THREADS) {
        const int c = channel(e);
        float acc = 0.f;
        if (c >= 0) {
            const float now = row[c];
            acc = fmaf(cw[(size_t)(taps - 1) * C_all + c], now, cb[c]);
            if (TAPS) {
                float w[TAPS ? TAPS : 1], u[TAPS ? TAPS : 1];
                #pragma unroll
                for (int j = 0; j < TAPS - 1; j++) {       // all loads first
                    const int back = TAPS - 1 - j, place = at >= back ? at - back : at - back + TAPS;
                    w[j] = cw[(size_t)j * C_all + c];
                    u[j] = back <= pos ? rg[(size_t)place * C_all + c] : 0.f;
                }
                #pragma unroll
                for (int j = 0; j < TAPS - 1; j++) acc = fmaf(w[j], u[j], acc);
            } else {
                for (int j = 0; j < taps - 1; j++) {
                    const int back = taps - 1 - j, place = at >= back ? at - back : at - back + taps;
                    if (back <= pos) acc = fmaf(cw[(size_t)j * C_all + c], rg[(size_t)place * C_all + c], acc);
                }
            }
        }
        sm[e] = __fdividef(acc, 1.0f + __expf(-acc));
    }
    const float dt = ik_softplusf(row[C_all + h] + dt_bias[h]), a = expf(A[h] * dt);
    __syncthreads();
    if (rg)                                                // the new inputs, behind every read of the ring in this block
        for (int e = threadIdx.x; e < (own_bc ? PT + 2 * N : PT); e += DEC_THREADS) {
            const int c = channel(e);
            if (c >= 0) rg[(size_t)at * C_all + c] = row[c];
        }
    const float4 x = *reinterpret_cast<const float4*>(sm + 4 * pv);
    const float4 xd = make_float4(dt * x.x, dt * x.y, dt * x.z, dt * x.w);
    const float* Bn = sm + PT;
    const float* Cn = Bn + N;
    float* sums = sm + PT + 2 * N;
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int n0 = 0; n0 < N; n0 += DEC_ROWS * slices) {
        if (n0) fetch(n0);
        #pragma unroll
        for (int r = 0; r < DEC_ROWS; r++) {
            const int n = n0 + slice + r * slices;
            if (n >= N) break;
            const float bn = Bn[n], cn = Cn[n];
            S[r].x = fmaf(a, S[r].x, bn * xd.x); y.x = fmaf(S[r].x, cn, y.x);
            S[r].y = fmaf(a, S[r].y, bn * xd.y); y.y = fmaf(S[r].y, cn, y.y);
            S[r].z = fmaf(a, S[r].z, bn * xd.z); y.z = fmaf(S[r].z, cn, y.z);
            S[r].w = fmaf(a, S[r].w, bn * xd.w); y.w = fmaf(S[r].w, cn, y.w);
            if (live) *reinterpret_cast<float4*>(st_out + (size_t)n * P) = S[r];
        }
    }
    // the slices' sums: sums [slices][PT] lies behind B and C, on a 16-byte boundary only when N is even; store one by one
    sums[slice * PT + 4 * pv] = y.x; sums[slice * PT + 4 * pv + 1] = y.y;
    sums[slice * PT + 4 * pv + 2] = y.z; sums[slice * PT + 4 * pv + 3] = y.w;
    __syncthreads();
    for (int e = threadIdx.x; e < PT; e += DEC_THREADS) {
        if (p0 + e >= P) continue;
        float o = 0.f;
        for (int s = 0; s < slices; s++) o += sums[s * PT + e];
        out[(size_t)tok * H * P + h * P + p0 + e] = fmaf(Dv[h], sm[e], o);
    }
}

// ------------------------------------------------------------------ gate, then an RMS norm in equal parts of the row
// out[t, i] = g_i / sqrt(mean over its part(g^2) + eps) * w[i] with g = x * silu(z), parts of d neighbouring values.  THREADS
// threads per part (32: a warp each, eight parts a block).  The part's g stays in registers (four values times KEEP a thread)
// where it fits.
template <typename TO> __device__ __forceinline__ float gate(float z) {       // silu; for 16-bit results with the hardware's exponential
    return sizeof(TO) == 2 ? __fdividef(z, 1.0f + __expf(-z)) : ik_siluf(z);
}
template <typename TO, int THREADS, bool VEC>
__global__ void __launch_bounds__(256)
gated_group_norm_kernel(const float* __restrict__ x, const float* __restrict__ z, int ldz, const float* __restrict__ w,
                        TO* __restrict__ out, int rows, int groups, int d, float eps) {
    constexpr int KEEP = 8, PB = 256 / THREADS;
    __shared__ float red[32];
    ik_pdl_wait();
    IK_AFTER_WAIT(x);
    IK_AFTER_WAIT(z);
    ik_pdl_launch_dependents();
    const int part = blockIdx.x * PB + threadIdx.x / THREADS, tid = threadIdx.x % THREADS;
    if (part >= rows * groups) return;                     // whole warps (THREADS 32) or whole blocks
    const int t = part / groups, gr = part - t * groups;
    const float* a = x + (size_t)part * d;
    const float* zz = z + (size_t)t * ldz + (size_t)gr * d;
    const float* ww = w + (size_t)gr * d;
    float ss = 0.f;
    auto total = [&](float v) -> float {
        if constexpr (THREADS == 256) {
            return ik_block_sum<256>(v, red);
        } else {
            #pragma unroll
            for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
            return v;
        }
    };
    if (VEC) {
        const int n4 = d >> 2;
        float4 g[KEEP];
        #pragma unroll
        for (int k = 0; k < KEEP; k++) {
            const int i = tid + k * THREADS;
            if (i < n4) {
                const float4 v = ik_ld4(a, 4 * (size_t)i), q = ik_ld4(zz, 4 * (size_t)i);
                g[k] = make_float4(v.x * gate<TO>(q.x), v.y * gate<TO>(q.y), v.z * gate<TO>(q.z), v.w * gate<TO>(q.w));
                ss = fmaf(g[k].x, g[k].x, fmaf(g[k].y, g[k].y, fmaf(g[k].z, g[k].z, fmaf(g[k].w, g[k].w, ss))));
            }
        }
        for (int i = tid + KEEP * THREADS; i < n4; i += THREADS) {
            const float4 v = ik_ld4(a, 4 * (size_t)i), q = ik_ld4(zz, 4 * (size_t)i);
            const float4 e = make_float4(v.x * gate<TO>(q.x), v.y * gate<TO>(q.y), v.z * gate<TO>(q.z), v.w * gate<TO>(q.w));
            ss = fmaf(e.x, e.x, fmaf(e.y, e.y, fmaf(e.z, e.z, fmaf(e.w, e.w, ss))));
        }
        const float s = 1.0f / sqrtf(total(ss) / (float)d + eps);
        #pragma unroll
        for (int k = 0; k < KEEP; k++) {
            const int i = tid + k * THREADS;
            if (i < n4) {
                const float4 q = ik_ld4(ww, 4 * (size_t)i);
                ik_st4(out, (size_t)part * d + 4 * (size_t)i, make_float4(g[k].x * s * q.x, g[k].y * s * q.y, g[k].z * s * q.z, g[k].w * s * q.w));
            }
        }
        for (int i = tid + KEEP * THREADS; i < n4; i += THREADS) {
            const float4 v = ik_ld4(a, 4 * (size_t)i), q = ik_ld4(zz, 4 * (size_t)i), c = ik_ld4(ww, 4 * (size_t)i);
            ik_st4(out, (size_t)part * d + 4 * (size_t)i, make_float4(v.x * gate<TO>(q.x) * s * c.x, v.y * gate<TO>(q.y) * s * c.y,
                                                                      v.z * gate<TO>(q.z) * s * c.z, v.w * gate<TO>(q.w) * s * c.w));
        }
    } else {
        for (int i = tid; i < d; i += THREADS) { const float v = a[i] * gate<TO>(zz[i]); ss = fmaf(v, v, ss); }
        const float s = 1.0f / sqrtf(total(ss) / (float)d + eps);
        for (int i = tid; i < d; i += THREADS) ik_st(out, (size_t)part * d + i, a[i] * gate<TO>(zz[i]) * s * ww[i]);
    }
}

template <typename TO>
int launch_gated_group_norm(const float* x, const float* z, int ldz, const float* w, TO* out, int rows, int groups, int d, float eps,
                            cudaStream_t stream) {
    const bool vec = d % 4 == 0 && ldz % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)z % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)out % 16 == 0;
    const int parts = rows * groups;
    if (d <= 512) {
        if (vec) IK_RETURN_IF_ERROR(ik_launch(gated_group_norm_kernel<TO, 32, true>, (parts + 7) / 8, 256, 0, stream, x, z, ldz, w, out, rows, groups, d, eps));
        else IK_RETURN_IF_ERROR(ik_launch(gated_group_norm_kernel<TO, 32, false>, (parts + 7) / 8, 256, 0, stream, x, z, ldz, w, out, rows, groups, d, eps));
    } else {
        if (vec) IK_RETURN_IF_ERROR(ik_launch(gated_group_norm_kernel<TO, 256, true>, parts, 256, 0, stream, x, z, ldz, w, out, rows, groups, d, eps));
        else IK_RETURN_IF_ERROR(ik_launch(gated_group_norm_kernel<TO, 256, false>, parts, 256, 0, stream, x, z, ldz, w, out, rows, groups, d, eps));
    }
    IK_LAUNCH_STATUS();
}

template <int NP, int NW>
int launch_chunk(const void* u, int ldu, const float* p, int ldp, int dt_off, const float* dt_bias, const float* A, const float* Dv,
                 float* state, const int* slots, const int* cu_seqlens, const int* kv_lens, float* out, int B, int H, int G, int N, int P,
                 cudaStream_t stream) {
    constexpr size_t smem = ssd_chunk_smem<NP, NW>();
    static bool raised = false;
    if (smem > 48 * 1024 && !raised) {
        IK_RETURN_IF_ERROR(cudaFuncSetAttribute(ssd_chunk_kernel<NP, NW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        raised = true;
    }
    const dim3 grid(H, B, (P + 16 * NW - 1) / (16 * NW));
    IK_RETURN_IF_ERROR(ik_launch(ssd_chunk_kernel<NP, NW>, grid, 32 * NW, smem, stream, (const bf16*)u, ldu, p, ldp, dt_off, dt_bias, A, Dv,
                                 state, slots, cu_seqlens, kv_lens, out, H, G, N, P));
    IK_LAUNCH_STATUS();
}

}  // namespace

// kind 0: token by token; kind 1: chunks on the tensor cores (bfloat16 u; N <= 128, N and P multiples of 8, aligned rows).
IK_EXPORT int ik_ssd(int kind, const void* u, int u_dtype, int ldu, const float* p, int ldp, int dt_off, const float* dt_bias,
                     const float* A, const float* Dv, float* state, const int* slots, const int* cu_seqlens, const int* kv_lens,
                     float* out, int T, int B, int H, int G, int N, int P, int exact, cudaStream_t stream) {
    if (T < 0 || B < 0 || H <= 0 || G <= 0 || H % G || N <= 0 || P <= 0 || !state || !A || !Dv || !dt_bias || ldu < H * P + 2 * G * N ||
        dt_off < 0 || ldp < dt_off + H || H > 65535 || B > 65535)
        return IK_BAD_ARGUMENT;
    if (T == 0 || B == 0) return IK_OK;
    if (kind == 1) {
        if (u_dtype != IK_BF16 || N > 128 || N % 8 || P % 8 || ldu % 8 || (uintptr_t)u % 16) return IK_UNSUPPORTED;
#define IK_CHUNK(NP)                                                                                                                       \
    return P <= 16 ? launch_chunk<NP, 1>(u, ldu, p, ldp, dt_off, dt_bias, A, Dv, state, slots, cu_seqlens, kv_lens, out, B, H, G, N, P, stream)     \
         : P <= 32 ? launch_chunk<NP, 2>(u, ldu, p, ldp, dt_off, dt_bias, A, Dv, state, slots, cu_seqlens, kv_lens, out, B, H, G, N, P, stream)     \
                   : launch_chunk<NP, 4>(u, ldu, p, ldp, dt_off, dt_bias, A, Dv, state, slots, cu_seqlens, kv_lens, out, B, H, G, N, P, stream)
        if (N <= 16) IK_CHUNK(16);
        if (N <= 32) IK_CHUNK(32);
        if (N <= 64) IK_CHUNK(64);
        IK_CHUNK(128);
#undef IK_CHUNK
    }
    int parts = (N + 7) / 8;
    if (parts > 16) parts = 16;
    const int R = (N + parts - 1) / parts, W = 2 * N + 34;
    if (R > 32) return IK_UNSUPPORTED;                     // up to 512 states
    const size_t smem = (size_t)(SCAN_TT * W + SCAN_TT * parts * 32) * sizeof(float);
    if (smem > 200 * 1024) return IK_UNSUPPORTED;
    const dim3 grid(B, H, (P + 31) / 32), block(32, parts);
#define IK_SCAN(TU, RMAX)                                                                                                                   \
    do {                                                                                                                                    \
        static bool raised = false;                                                                                                         \
        if (smem > 48 * 1024 && !raised) {                                                                                                  \
            IK_RETURN_IF_ERROR(cudaFuncSetAttribute(ssd_scan_kernel<TU, RMAX>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));   \
            raised = true;                                                                                                                  \
        }                                                                                                                                   \
        IK_RETURN_IF_ERROR(ik_launch(ssd_scan_kernel<TU, RMAX>, grid, block, smem, stream, (const TU*)u, ldu, p, ldp, dt_off, dt_bias, A, Dv, \
                                     state, slots, cu_seqlens, kv_lens, out, H, G, N, P, R, exact));                                        \
    } while (0)
    if (u_dtype == IK_F32) { if (R <= 8) IK_SCAN(float, 8); else if (R <= 16) IK_SCAN(float, 16); else IK_SCAN(float, 32); }
    else if (u_dtype == IK_BF16) { if (R <= 8) IK_SCAN(bf16, 8); else if (R <= 16) IK_SCAN(bf16, 16); else IK_SCAN(bf16, 32); }
    else return IK_BAD_ARGUMENT;
#undef IK_SCAN
    IK_LAUNCH_STATUS();
}

// One token per sequence: convolution (taps, cw tap-major, bias cb, ring of taps inputs) and the step of the recurrence.  The
// columns of p: x, B, C from x_off, then one raw step per head.  P a multiple of 4.
IK_EXPORT int ik_ssd_decode(const float* p, int ldp, int x_off, const float* cw, const float* cb, float* ring, const float* dt_bias,
                            const float* A, const float* Dv, float* state, const int* slots, const int* cu_seqlens, const int* kv_lens,
                            float* out, int B, int H, int G, int N, int P, int taps, cudaStream_t stream) {
    if (B < 0 || H <= 0 || G <= 0 || H % G || N <= 0 || P <= 0 || taps <= 0 || (taps > 1 && !ring) || !cw || !cb || !state || x_off < 0 ||
        ldp < x_off + H * P + 2 * G * N + H || H > 65535 || B > 65535)
        return IK_BAD_ARGUMENT;
    if (B == 0) return IK_OK;
    if (P % 4 || (uintptr_t)state % 16) return IK_UNSUPPORTED;
    int pv_n = 1;
    while (pv_n < 16 && 4 * pv_n < P) pv_n *= 2;
    const int PT = 4 * pv_n, slices = DEC_THREADS / pv_n;
    const size_t smem = (size_t)(PT + 2 * N + slices * PT) * sizeof(float);
    if (smem > 48 * 1024) return IK_UNSUPPORTED;
    const dim3 grid(H, B, (P + PT - 1) / PT);
#define IK_DEC(TAPS)                                                                                                                  \
    IK_RETURN_IF_ERROR(ik_launch(ssd_decode_kernel<TAPS>, grid, DEC_THREADS, smem, stream, p, ldp, x_off, cw, cb, taps > 1 ? ring : nullptr, dt_bias, \
                                 A, Dv, state, slots, cu_seqlens, kv_lens, out, H, G, N, P, taps, pv_n))
    switch (taps) {
        case 1: IK_DEC(1); break;
        case 2: IK_DEC(2); break;
        case 3: IK_DEC(3); break;
        case 4: IK_DEC(4); break;
        default: IK_DEC(0);
    }
#undef IK_DEC
    IK_LAUNCH_STATUS();
}

IK_EXPORT int ik_gated_group_norm(const float* x, const float* z, int ldz, const float* w, void* out, int out_dtype, int rows, int groups,
                                  int d, float eps, cudaStream_t stream) {
    if (rows < 0 || groups <= 0 || d <= 0 || !x || !z || !w || ldz < groups * d) return IK_BAD_ARGUMENT;
    if (rows == 0) return IK_OK;
    if (out_dtype == IK_F32) return launch_gated_group_norm<float>(x, z, ldz, w, (float*)out, rows, groups, d, eps, stream);
    if (out_dtype == IK_BF16) return launch_gated_group_norm<bf16>(x, z, ldz, w, (bf16*)out, rows, groups, d, eps, stream);
    return IK_BAD_ARGUMENT;
}
