// State-space duality for prompts on the fifth-generation tensor cores: the chunk form of ssd.cu (see there for the
// recurrence, its state and the sums) with chunks of 128 tokens, for 64 or 128 states and values in multiples of 64.
//
// A block owns 64 columns of one head's state for one sequence and walks the chunks in order.  With c_i the running sum of
// A dt, per chunk:
//   scores  Sc = C B^T                          [128 tokens x 128 tokens]   operands from shared memory
//   carry   Yi = C S                            [128 tokens x 64]           S as three bfloat16 terms in shared memory
//   own     Yp = P x,  P_ij = exp(c_i - c_j) dt_j Sc_ij for j <= i          P as two bfloat16 terms in TMEM
//   gain    D  = W x,  W_nj = exp(c_last - c_j) dt_j B_jn  [states x 64]    W as two bfloat16 terms in TMEM
//   y_i = exp(c_i) Yi_i + Yp_i + skip x_i,      S <- exp(c_last) S + D.
// x, B and C are bfloat16 as they come; a float operand is handed over as the sum of two bfloat16 numbers (relative error
// 2^-17; the state three: 2^-25), each with a product of its own, and all sums are float.  The state itself stays in registers as floats, one row (64
// columns) per thread.
//   warp 0        TMA: C, B, x of a chunk into one of two stages.
//   warps 1, 3    tcgen05.mma: scores and own tokens; gain and carry.  Issuing a product costs its thread more than the tensor
//                 core takes for one this narrow, so two threads issue.
//   warp 2        steps, running sums (in double, so that a difference of two sums is exact where the sums are large) and the
//                 factors made of them, a chunk ahead.
//   warps 4..7    a token per thread: P from the scores, y from the two results (to global memory by pieces of rows, through
//                 shared memory).  For columns j outside a warp's own 32 x 32
//                 diagonal block exp(c_i - c_j) is the product of two factors, of the row and of the column, both at most 1
//                 (c at the block's first row lies between the two), so only the diagonal block needs an exponential per element.
//   warps 8..11   a state per thread: S from D, and S as three terms.
//   warps 12..15  a state per thread: W from B and the factors.
// Every mbarrier here completes one phase per chunk (per use of a stage), and no phase can complete before every waiter has
// seen the one before it: see the notes at the arrivals.  All waits are bounded (tc_common.cuh); on a timeout the status word
// is set, the block leaves its loops and frees its TMEM.
#define IK_FAMILY 8
#include "common.cuh"
#include "tc_common.cuh"

namespace {

typedef __nv_bfloat16 bf16;

constexpr int Q = 128, PC = 64;                            // tokens a chunk, columns a block
constexpr int TILE_BYTES = Q * 128;                        // 128 rows of 64 bfloat16
constexpr int COL_SC = 0, COL_PL = 128, COL_WH = 192, COL_WL = 256, COL_YI = 320, COL_YP = 384, COL_D = 448;   // TMEM columns

struct Factors {                                           // what the decays of a chunk come to
    float ch[Q], cl[Q];                                    // c_i in powers of two, as the sum of two floats
    float dt[Q];
    float ei[Q];                                           // exp(c_i)
    float er[Q];                                           // exp(c_i - c at the row before i's block of 32)
    float w[Q];                                            // exp(c_last - c_j) dt_j
    float f[3][96];                                        // f[I - 1][j] = exp(c at the row before block I - c_j) dt_j, j < 32 I
    float keep, pad[3];                                    // exp(c_last)
};

template <int NS> constexpr int stage_bytes() { return (2 * (NS / 64) + 1) * TILE_BYTES; }      // C, B, x
constexpr int Y_BYTES = Q * 16 * 4;                         // y on its way out, 16 columns at a time
template <int NS> constexpr int smem_bytes() { return 2 * stage_bytes<NS>() + 3 * NS * 128 + Y_BYTES + 2 * (int)sizeof(Factors) + 256; }

// the leading bfloat16 parts of two floats, packed; the floats become what is left of them
__device__ __forceinline__ uint32_t take2(float& a, float& b) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    const uint32_t w = *reinterpret_cast<const uint32_t*>(&v);
    asm("{\n\t.reg .b64 x, y, m;\n\t"
        "mov.b64 x, {%0, %1};\n\t"
        "mov.b64 y, {%2, %3};\n\t"
        "mov.b64 m, {%4, %4};\n\t"
        "fma.rn.f32x2 x, y, m, x;\n\t"
        "mov.b64 {%0, %1}, x;\n\t}"
        : "+f"(a), "+f"(b) : "f"(__uint_as_float(w << 16)), "f"(__uint_as_float(w & 0xffff0000u)), "f"(-1.0f));
    return w;
}
// (a, b) *= (c, d)
__device__ __forceinline__ void mul2(float& a, float& b, float c, float d) {
    asm("{\n\t.reg .b64 x, y;\n\t"
        "mov.b64 x, {%0, %1};\n\t"
        "mov.b64 y, {%2, %3};\n\t"
        "mul.rn.f32x2 x, x, y;\n\t"
        "mov.b64 {%0, %1}, x;\n\t}"
        : "+f"(a), "+f"(b) : "f"(c), "f"(d));
}
__device__ __forceinline__ void store8(float* p, const float* v) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}

template <int NS>
__global__ void __launch_bounds__(512, 1)
ssd_tc_kernel(const __grid_constant__ CUtensorMap map_u, const float* __restrict__ p, int ldp, int dt_off, const float* __restrict__ dt_bias,
              const float* __restrict__ A, const float* __restrict__ Dv, float* __restrict__ state, const int* __restrict__ slots,
              const int* __restrict__ cu_seqlens, const int* __restrict__ kv_lens, float* __restrict__ out, int H, int G, int P, int* status) {
    extern __shared__ __align__(1024) unsigned char smem[];
    ik_pdl_wait();
    IK_AFTER_WAIT(p);
    IK_AFTER_WAIT(slots);
    IK_AFTER_WAIT(cu_seqlens);
    IK_AFTER_WAIT(kv_lens);
    constexpr int BOXES = NS / 64, SB = stage_bytes<NS>();
    const int h = blockIdx.x, b = blockIdx.y, p0 = blockIdx.z * PC;
    const int lo = cu_seqlens[b], hi = cu_seqlens[b + 1], end = kv_lens[b], start = end - (hi - lo);
    if (hi <= lo) return;
    if (ik_status_has(status, IK_STATUS_GEMM_TIMEOUT)) return;
    if (smem_u32(smem) & 1023) {                           // the swizzled tiles need it
        if (threadIdx.x == 0) ik_set_status(status, IK_STATUS_SMEM_ALIGN);
        return;
    }
    const int n_chunks = (hi - lo + Q - 1) / Q;
    unsigned char* Ss = smem + 2 * SB;                     // [3][NS rows][64 columns], swizzled like x
    unsigned char* Ys = Ss + 3 * NS * 128;
    Factors* fac = (Factors*)(Ys + Y_BYTES);               // [2]
    uint64_t* full = (uint64_t*)(fac + 2);                 // [2] a stage's tiles are there
    uint64_t* freed = full + 2;                            // [2] ... and have been read: two issuers' products, 128 + 128 threads
    uint64_t* fac_full = freed + 2;                        // [2]
    uint64_t* fac_free = fac_full + 2;                     // [2]
    uint64_t* sc_full = fac_free + 2;
    uint64_t* p_ready = sc_full + 1;
    uint64_t* w_ready = p_ready + 1;
    uint64_t* d_full = w_ready + 1;
    uint64_t* s_ready = d_full + 1;                        // the state before chunk c, as three terms
    uint64_t* yi_full = s_ready + 1;
    uint64_t* yp_full = yi_full + 1;
    uint64_t* y_read = yp_full + 1;                        // both have been read
    uint64_t* d_read = y_read + 1;
    uint32_t* tmem_slot = (uint32_t*)(d_read + 1);
    volatile int* abort_flag = (volatile int*)(tmem_slot + 1);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (int s = 0; s < 2; s++) {
            mbar_init(full + s, 1);
            mbar_init(freed + s, 258);
            mbar_init(fac_full + s, 32);
            mbar_init(fac_free + s, 384);
        }
        mbar_init(sc_full, 1);
        mbar_init(p_ready, 128);
        mbar_init(w_ready, 128);
        mbar_init(d_full, 1);
        mbar_init(s_ready, 128);
        mbar_init(yi_full, 1);
        mbar_init(yp_full, 1);
        mbar_init(y_read, 128);
        mbar_init(d_read, 128);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("prefetch.tensormap [%0];" :: "l"(&map_u) : "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" :: "r"(smem_u32(tmem_slot)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot;
    const int grp = h / (H / G);
    const unsigned long long lim = IK_WAIT_LIMIT_NS;

    if (warp == 0) {
        if (lane == 0) {
            const int x_off = h * P + p0, b_off = H * P + grp * NS, c_off = H * P + G * NS + grp * NS;
            for (int c = 0; c < n_chunks; c++) {
                const int s = c & 1;
                if (!mbar_wait(freed + s, ((c >> 1) & 1) ^ 1, abort_flag, status, lim, 31, c)) break;
                unsigned char* st = smem + s * SB;
                mbar_expect_tx(full + s, SB);
                for (int k = 0; k < BOXES; k++) tma_load_2d(st + k * TILE_BYTES, &map_u, c_off + k * 64, lo + c * Q, full + s);
                for (int k = 0; k < BOXES; k++) tma_load_2d(st + (BOXES + k) * TILE_BYTES, &map_u, b_off + k * 64, lo + c * Q, full + s);
                tma_load_2d(st + 2 * BOXES * TILE_BYTES, &map_u, x_off, lo + c * Q, full + s);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t id_sc = umma_idesc(Q), id_v = umma_idesc(PC, 1);
            for (int c = 0; c < n_chunks; c++) {
                const int s = c & 1;
                const uint32_t c_addr = smem_u32(smem + s * SB), b_addr = c_addr + BOXES * TILE_BYTES, x_addr = b_addr + BOXES * TILE_BYTES;
                if (!mbar_wait(full + s, (c >> 1) & 1, abort_flag, status, lim, 32, c)) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                // the scores overwrite the P of the chunk before, whose products were issued before these
                #pragma unroll
                for (int j = 0; j < NS / 16; j++)
                    umma(tmem + COL_SC, umma_desc(c_addr + (j / 4) * TILE_BYTES + (j % 4) * 32), umma_desc(b_addr + (j / 4) * TILE_BYTES + (j % 4) * 32),
                         id_sc, j != 0);
                umma_commit(sc_full);
                if (!mbar_wait(p_ready, c & 1, abort_flag, status, lim, 34, c)) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                #pragma unroll
                for (int j = 0; j < Q / 16; j++) {
                    const uint64_t xd = umma_desc_mn(x_addr + j * 2048, TILE_BYTES);
                    umma_ts(tmem + COL_YP, tmem + COL_PL + j * 8, xd, id_v, j != 0);
                    umma_ts(tmem + COL_YP, tmem + COL_SC + j * 8, xd, id_v, 1);
                }
                umma_commit(yp_full);
                if (c + 2 < n_chunks) umma_commit(freed + s);          // (nobody waits for the last two)
            }
        }
    } else if (warp == 3) {
        if (lane == 0) {
            const uint32_t id_v = umma_idesc(PC, 1), s_addr = smem_u32(Ss);
            for (int c = 0; c < n_chunks; c++) {
                const int s = c & 1;
                const uint32_t c_addr = smem_u32(smem + s * SB), x_addr = c_addr + 2 * BOXES * TILE_BYTES;
                if (!mbar_wait(full + s, (c >> 1) & 1, abort_flag, status, lim, 32, c)) break;
                // the state's terms, and the carry of the chunk before read from its accumulator
                if (!mbar_wait(s_ready, c & 1, abort_flag, status, lim, 35, c) || !mbar_wait(y_read, (c & 1) ^ 1, abort_flag, status, lim, 45, c)) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                #pragma unroll
                for (int e = 2; e >= 0; e--)
                    #pragma unroll
                    for (int j = 0; j < NS / 16; j++)
                        umma(tmem + COL_YI, umma_desc(c_addr + (j / 4) * TILE_BYTES + (j % 4) * 32), umma_desc_mn(s_addr + e * NS * 128 + j * 2048, NS * 128),
                             id_v, e != 2 || j != 0);
                umma_commit(yi_full);
                if (!mbar_wait(w_ready, c & 1, abort_flag, status, lim, 33, c) || !mbar_wait(d_read, (c & 1) ^ 1, abort_flag, status, lim, 48, c)) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                #pragma unroll
                for (int j = 0; j < Q / 16; j++) {
                    const uint64_t xd = umma_desc_mn(x_addr + j * 2048, TILE_BYTES);
                    umma_ts(tmem + COL_D, tmem + COL_WL + j * 8, xd, id_v, j != 0);
                    umma_ts(tmem + COL_D, tmem + COL_WH + j * 8, xd, id_v, 1);
                }
                umma_commit(d_full);
                if (c + 2 < n_chunks) umma_commit(freed + s);          // (nobody waits for the last two)
            }
        }
    } else if (warp == 2) {
        // lane l: tokens 4l .. 4l + 3 of the chunk
        const double rate2 = (double)A[h] * 1.4426950408889634;
        const float bias = dt_bias[h];
        float raw[4];
        auto fetch = [&](int c) {
            #pragma unroll
            for (int k = 0; k < 4; k++) {
                const int t = lo + c * Q + 4 * lane + k;
                raw[k] = t < hi ? p[(size_t)t * ldp + dt_off + h] : 0.f;
            }
        };
        fetch(0);
        for (int c = 0; c < n_chunks; c++) {
            if (!mbar_wait(fac_free + (c & 1), ((c >> 1) & 1) ^ 1, abort_flag, status, lim, 36, c)) break;
            Factors& F = fac[c & 1];
            float dt[4];
            double cs[4], run = 0.0;
            #pragma unroll
            for (int k = 0; k < 4; k++) {
                const float z = raw[k] + bias;
                dt[k] = lo + c * Q + 4 * lane + k < hi ? (z > 20.0f ? z : log1pf(expf(z))) : 0.f;
                run += rate2 * (double)dt[k];
                cs[k] = run;
            }
            if (c + 1 < n_chunks) fetch(c + 1);
            double inc = run;
            #pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const double q = __shfl_up_sync(0xffffffffu, inc, o);
                if (lane >= o) inc += q;
            }
            const double before = inc - run;
            #pragma unroll
            for (int k = 0; k < 4; k++) cs[k] += before;
            const double last = __shfl_sync(0xffffffffu, cs[3], 31);
            double ref[3];
            #pragma unroll
            for (int I = 1; I < 4; I++) ref[I - 1] = __shfl_sync(0xffffffffu, cs[3], 8 * I - 1);
            const int mine = lane >> 3;                    // the block of 32 rows these tokens lie in
            const double my_ref = mine == 0 ? 0.0 : mine == 1 ? ref[0] : mine == 2 ? ref[1] : ref[2];
            #pragma unroll
            for (int k = 0; k < 4; k++) {
                const int j = 4 * lane + k;
                const float c_hi = (float)cs[k];
                F.ch[j] = c_hi;
                F.cl[j] = (float)(cs[k] - (double)c_hi);
                F.dt[j] = dt[k];
                F.ei[j] = ik_ex2(c_hi);
                F.er[j] = ik_ex2((float)(cs[k] - my_ref));
                F.w[j] = ik_ex2((float)(last - cs[k])) * dt[k];
                #pragma unroll
                for (int I = 1; I < 4; I++)
                    if (j < 32 * I) F.f[I - 1][j] = ik_ex2((float)(ref[I - 1] - cs[k])) * dt[k];
            }
            if (lane == 0) F.keep = ik_ex2((float)last);
            mbar_arrive(fac_full + (c & 1));
        }
    } else if (warp >= 4 && warp < 8) {
        const int quarter = warp & 3, i = quarter * 32 + lane;
        const uint32_t base = tmem + ((uint32_t)(quarter * 32) << 16);
        const float skip = Dv[h];
        unsigned char* ys = Ys + quarter * 2048;             // 32 rows of 16 floats, 16-byte pieces swizzled within eight rows
        bool ok = true;
        for (int c = 0; c < n_chunks; c++) {
            const int s = c & 1;
            ok = mbar_wait(fac_full + s, (c >> 1) & 1, abort_flag, status, lim, 37, c) && mbar_wait(sc_full, c & 1, abort_flag, status, lim, 38, c);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const Factors& F = fac[s];
            const float my_er = F.er[i], my_ei = F.ei[i];
            #pragma unroll 1
            for (int k = 0; k < 4; k++) {                  // 32 columns a turn; P lies over scores that have been read
                uint32_t ph[16], pl[16];
                if (k > quarter) {
                    #pragma unroll
                    for (int e = 0; e < 16; e++) ph[e] = pl[e] = 0u;
                } else {
                    float v[32];
                    tmem_ld16_issue(base + COL_SC + 32 * k, v);
                    tmem_ld16_issue(base + COL_SC + 32 * k + 16, v + 16);
                    tmem_ld_wait();
                    if (k < quarter) {
                        const float4* f = reinterpret_cast<const float4*>(F.f[quarter - 1] + 32 * k);
                        #pragma unroll
                        for (int e = 0; e < 8; e++) {
                            const float4 q = f[e];
                            mul2(v[4 * e], v[4 * e + 1], q.x, q.y);
                            mul2(v[4 * e + 2], v[4 * e + 3], q.z, q.w);
                            mul2(v[4 * e], v[4 * e + 1], my_er, my_er);
                            mul2(v[4 * e + 2], v[4 * e + 3], my_er, my_er);
                        }
                    } else {
                        const float ch = F.ch[i], cl = F.cl[i];
                        const float4* ch4 = reinterpret_cast<const float4*>(F.ch + 32 * k);
                        const float4* cl4 = reinterpret_cast<const float4*>(F.cl + 32 * k);
                        const float4* dt4 = reinterpret_cast<const float4*>(F.dt + 32 * k);
                        #pragma unroll
                        for (int e = 0; e < 8; e++) {
                            const float4 a = ch4[e], q = cl4[e], d = dt4[e];
                            const float aa[4] = {a.x, a.y, a.z, a.w}, qq[4] = {q.x, q.y, q.z, q.w}, dd[4] = {d.x, d.y, d.z, d.w};
                            #pragma unroll
                            for (int r = 0; r < 4; r++)
                                v[4 * e + r] = 4 * e + r <= lane ? v[4 * e + r] * (ik_ex2((ch - aa[r]) + (cl - qq[r])) * dd[r]) : 0.f;
                        }
                    }
                    #pragma unroll
                    for (int e = 0; e < 16; e++) {
                        ph[e] = take2(v[2 * e], v[2 * e + 1]);
                        pl[e] = take2(v[2 * e], v[2 * e + 1]);
                    }
                }
                tmem_st16_bits(base + COL_SC + 16 * k, ph);
                tmem_st16_bits(base + COL_PL + 16 * k, pl);
            }
            tmem_st_wait();
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(fac_free + s);
            mbar_arrive(p_ready);                          // (this thread has read the y of the chunk before)
            ok = mbar_wait(yi_full, c & 1, abort_flag, status, lim, 39, c) && mbar_wait(yp_full, c & 1, abort_flag, status, lim, 39, c) &&
                 mbar_wait(full + s, (c >> 1) & 1, abort_flag, status, lim, 40, c);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const unsigned char* xrow = smem + s * SB + 2 * BOXES * TILE_BYTES + i * 128;
            const int t0 = lo + c * Q + 32 * quarter;
            float ahead[2][16];                            // the next turn's results are asked for a turn early
            tmem_ld16_issue(base + COL_YI, ahead[0]);
            tmem_ld16_issue(base + COL_YP, ahead[1]);
            #pragma unroll
            for (int k = 0; k < 4; k++) {                  // 16 columns a turn
                float yi[16], yp[16];
                tmem_ld_wait();
                #pragma unroll
                for (int e = 0; e < 16; e++) { yi[e] = ahead[0][e]; yp[e] = ahead[1][e]; }
                if (k < 3) {
                    tmem_ld16_issue(base + COL_YI + 16 * (k + 1), ahead[0]);
                    tmem_ld16_issue(base + COL_YP + 16 * (k + 1), ahead[1]);
                }
                #pragma unroll
                for (int e = 0; e < 2; e++) {
                    const uint4 xv = *reinterpret_cast<const uint4*>(xrow + (((2 * k + e) ^ (i & 7)) << 4));
                    const uint32_t xw[4] = {xv.x, xv.y, xv.z, xv.w};
                    #pragma unroll
                    for (int q = 0; q < 4; q++) {
                        const int a = 8 * e + 2 * q;
                        yp[a] = fmaf(my_ei, yi[a], fmaf(skip, __uint_as_float(xw[q] << 16), yp[a]));
                        yp[a + 1] = fmaf(my_ei, yi[a + 1], fmaf(skip, __uint_as_float(xw[q] & 0xffff0000u), yp[a + 1]));
                    }
                    #pragma unroll
                    for (int q = 0; q < 2; q++)
                        *reinterpret_cast<float4*>(ys + lane * 64 + (((2 * e + q) ^ ((lane >> 1) & 3)) << 4)) =
                            make_float4(yp[8 * e + 4 * q], yp[8 * e + 4 * q + 1], yp[8 * e + 4 * q + 2], yp[8 * e + 4 * q + 3]);
                }
                if (k == 3) {                              // all of this chunk's results and x have been read
                    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
                    mbar_arrive(y_read);
                    mbar_arrive(freed + s);
                }
                __syncwarp();
                #pragma unroll
                for (int r8 = 0; r8 < 4; r8++) {           // eight rows of 64 bytes an instruction
                    const int r = 8 * r8 + (lane >> 2), piece = lane & 3;
                    const float4 v = *reinterpret_cast<const float4*>(ys + r * 64 + ((piece ^ ((r >> 1) & 3)) << 4));
                    if (t0 + r < hi) *reinterpret_cast<float4*>(out + (size_t)(t0 + r) * H * P + h * P + p0 + 16 * k + 4 * piece) = v;
                }
                __syncwarp();
            }
        }
    } else if (warp >= 8 && warp < 12) {
        const int quarter = warp & 3, n = quarter * 32 + lane;
        const bool live = n < NS;
        const uint32_t base = tmem + ((uint32_t)(quarter * 32) << 16);
        const size_t per = (size_t)H * NS * P, at = (size_t)h * NS * P + (size_t)(live ? n : 0) * P + p0;
        const float* st_in = state + ((size_t)slots[b] * 2 + ((start - 1) & 1)) * per + at;
        float* st_out = state + ((size_t)slots[b] * 2 + ((end - 1) & 1)) * per + at;
        float S[PC];
        #pragma unroll
        for (int k = 0; k < PC / 4; k++) {
            const float4 v = live && start > 0 ? reinterpret_cast<const float4*>(st_in)[k] : make_float4(0.f, 0.f, 0.f, 0.f);
            S[4 * k] = v.x; S[4 * k + 1] = v.y; S[4 * k + 2] = v.z; S[4 * k + 3] = v.w;
        }
        // the state as three terms, a row of 64 columns each; 16-byte pieces swizzled within groups of eight rows
        auto publish = [&]() {
            if (live) {
                unsigned char* row = Ss + n * 128;
                #pragma unroll
                for (int k = 0; k < 8; k++) {
                    uint32_t t0[4], t1[4], t2[4];
                    #pragma unroll
                    for (int q = 0; q < 4; q++) {
                        float a = S[8 * k + 2 * q], d = S[8 * k + 2 * q + 1];
                        t0[q] = take2(a, d);
                        t1[q] = take2(a, d);
                        t2[q] = take2(a, d);
                    }
                    const int o = (k ^ (n & 7)) << 4;
                    *reinterpret_cast<uint4*>(row + o) = make_uint4(t0[0], t0[1], t0[2], t0[3]);
                    *reinterpret_cast<uint4*>(row + NS * 128 + o) = make_uint4(t1[0], t1[1], t1[2], t1[3]);
                    *reinterpret_cast<uint4*>(row + 2 * NS * 128 + o) = make_uint4(t2[0], t2[1], t2[2], t2[3]);
                }
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            mbar_arrive(s_ready);
        };
        publish();
        bool ok = true;
        for (int c = 0; c < n_chunks; c++) {
            const int s = c & 1;
            ok = mbar_wait(fac_full + s, (c >> 1) & 1, abort_flag, status, lim, 41, c);
            if (!ok) break;
            const float keep = fac[s].keep;
            mbar_arrive(fac_free + s);
            // D, and the carry's product, which still reads the terms of the state before
            ok = mbar_wait(d_full, c & 1, abort_flag, status, lim, 43, c) && mbar_wait(yi_full, c & 1, abort_flag, status, lim, 44, c);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            if (quarter * 32 < NS) {
                #pragma unroll
                for (int k = 0; k < PC / 32; k++) {
                    float d[32];
                    tmem_ld16_issue(base + COL_D + 32 * k, d);
                    tmem_ld16_issue(base + COL_D + 32 * k + 16, d + 16);
                    tmem_ld_wait();
                    #pragma unroll
                    for (int e = 0; e < 32; e++) S[32 * k + e] = fmaf(keep, S[32 * k + e], d[e]);
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(d_read);
            if (c + 1 < n_chunks) publish();
        }
        if (ok && live) {
            #pragma unroll
            for (int k = 0; k < PC / 8; k++) store8(st_out + 8 * k, S + 8 * k);
        }
    } else if (warp >= 12) {
        const int quarter = warp & 3, n = quarter * 32 + lane;
        const uint32_t base = tmem + ((uint32_t)(quarter * 32) << 16);
        if (n >= NS) {                                     // rows of W beyond the states: zeros for good
            const uint32_t z[16] = {};
            for (int k = 0; k < 4; k++) {
                tmem_st16_bits(base + COL_WH + 16 * k, z);
                tmem_st16_bits(base + COL_WL + 16 * k, z);
            }
            tmem_st_wait();
        }
        for (int c = 0; c < n_chunks; c++) {
            const int s = c & 1;
            // (the gain's product of the chunk before has read its W)
            if (!mbar_wait(fac_full + s, (c >> 1) & 1, abort_flag, status, lim, 46, c) || !mbar_wait(full + s, (c >> 1) & 1, abort_flag, status, lim, 42, c) ||
                (c > 0 && !mbar_wait(d_full, (c - 1) & 1, abort_flag, status, lim, 47, c)))
                break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const Factors& F = fac[s];
            if (quarter * 32 < NS) {
                const unsigned char* bt = smem + s * SB + (BOXES + n / 64) * TILE_BYTES;      // 128 tokens x 64 states
                const int piece = (n & 63) >> 3, in = (n & 7) * 2;
                #pragma unroll 1
                for (int k = 0; k < 4; k++) {              // 32 tokens a turn
                    float v[32];
                    const float4* w4 = reinterpret_cast<const float4*>(F.w + 32 * k);
                    #pragma unroll
                    for (int e = 0; e < 8; e++) {
                        const float4 q = w4[e];
                        #pragma unroll
                        for (int r = 0; r < 4; r++) {
                            const int j = 32 * k + 4 * e + r;      // j & 7 is known: 32 k is a multiple of eight
                            const unsigned short raw = *reinterpret_cast<const unsigned short*>(bt + j * 128 + ((piece ^ ((4 * e + r) & 7)) << 4) + in);
                            v[4 * e + r] = __uint_as_float((uint32_t)raw << 16);
                        }
                        mul2(v[4 * e], v[4 * e + 1], q.x, q.y);
                        mul2(v[4 * e + 2], v[4 * e + 3], q.z, q.w);
                    }
                    uint32_t wh[16], wl[16];
                    #pragma unroll
                    for (int e = 0; e < 16; e++) {
                        wh[e] = take2(v[2 * e], v[2 * e + 1]);
                        wl[e] = take2(v[2 * e], v[2 * e + 1]);
                    }
                    tmem_st16_bits(base + COL_WH + 16 * k, wh);
                    tmem_st16_bits(base + COL_WL + 16 * k, wl);
                }
                tmem_st_wait();
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(freed + s);
            mbar_arrive(fac_free + s);
            mbar_arrive(w_ready);
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" :: "r"(tmem), "r"(512u) : "memory");
    }
}

template <int NS>
int launch(const CUtensorMap& map, const float* p, int ldp, int dt_off, const float* dt_bias, const float* A, const float* Dv, float* state,
           const int* slots, const int* cu_seqlens, const int* kv_lens, float* out, int B, int H, int G, int P, int* status, cudaStream_t stream) {
    constexpr int smem = smem_bytes<NS>();
    static bool raised = false;
    if (!raised) {
        IK_RETURN_IF_ERROR(cudaFuncSetAttribute(ssd_tc_kernel<NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        raised = true;
    }
    IK_RETURN_IF_ERROR(ik_launch(ssd_tc_kernel<NS>, dim3(H, B, P / PC), 512, smem, stream, map, p, ldp, dt_off, dt_bias, A, Dv, state, slots,
                                 cu_seqlens, kv_lens, out, H, G, P, status));
    IK_LAUNCH_STATUS();
}

}  // namespace

// Sites of this module's waits: 31 loader for a free stage; 32 issuers for a stage, 33 W, 34 P, 35 the state's terms, 45 the
// carry's accumulator, 48 the gain's; 36 factors
// for a free place; 37..40 token threads for factors, scores, results, the stage; 41, 43, 44 state threads for factors, the gain, the
// carry; 42, 46, 47 W threads for the stage, factors, the gain before.
IK_EXPORT int ik_ssd_take_wait_record(int* out4) { return ik_take_wait_record(out4); }

// Arguments as ik_ssd's (ssd.cu); bfloat16 u, N 64 or 128, P a multiple of 64, 16-byte aligned rows.
IK_EXPORT int ik_ssd_tcgen05(const void* u, int ldu, const float* p, int ldp, int dt_off, const float* dt_bias, const float* A, const float* Dv,
                             float* state, const int* slots, const int* cu_seqlens, const int* kv_lens, float* out, int T, int B, int H, int G,
                             int N, int P, int* status, cudaStream_t stream) {
    if (T < 0 || B < 0 || H <= 0 || G <= 0 || H % G || N <= 0 || P <= 0 || !state || !A || !Dv || !dt_bias || ldu < H * P + 2 * G * N ||
        dt_off < 0 || ldp < dt_off + H || B > 65535)
        return IK_BAD_ARGUMENT;
    if (T == 0 || B == 0) return IK_OK;
    if ((N != 64 && N != 128) || P % PC || ldu % 8 || (uintptr_t)u % 16 || (uintptr_t)state % 16 || (uintptr_t)out % 16) return IK_UNSUPPORTED;
    CUtensorMap map;
    const int st = ik_make_map(&map, u, (unsigned long long)T, H * P + 2 * G * N, (unsigned long long)ldu, Q);
    if (st != IK_OK) return st;
    if (N == 64) return launch<64>(map, p, ldp, dt_off, dt_bias, A, Dv, state, slots, cu_seqlens, kv_lens, out, B, H, G, P, status, stream);
    return launch<128>(map, p, ldp, dt_off, dt_bias, A, Dv, state, slots, cu_seqlens, kv_lens, out, B, H, G, P, status, stream);
}
