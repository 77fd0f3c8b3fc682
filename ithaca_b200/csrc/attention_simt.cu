// Attention over the paged cache on the CUDA cores, for prefill and decode alike.
//
// One block per (query token, head).  Keys run from j0 to the token's own position
// (causal by loop bound; j0 > 0 only under a window), in tiles of 128 that start at
// absolute multiples of 128 (the tiles of the first `keep` keys, which stay visible behind the window, come first), so the order in which a query's keys are reduced depends
// only on its position, not on how the tokens were cut into steps or batched.
// Scores, the running maximum, the sum and the output are float; exp is the accurate
// function.  This is the 32-bit path's attention and the fallback for head sizes the
// tensor-core kernels do not take.  Options: a cap on the scores, s <- cap * tanh(s / cap) after the scale
// (cap 0 = none), value heads of another size than the key heads (hdv), values that are the leading hdv columns of the
// key rows themselves (v_pages = k_pages with ldv = hd: a latent that serves as key and value), and a sink: one more
// key of score 0 that carries no value, so that the weights are exp(s_j) / (1 + sum exp(s_j)).  Under a window the first
// `keep` keys of the sequence may stay visible to every later query.  With key_scales (scales[page][kv head][position in page])
// every score is multiplied by its key's number, for keys that are stored as projected because they are the values too and whose
// norm is a factor.  With slopes [nh] a score loses slope * (i - j), behind the cap.
#include <math.h>
#define IK_FAMILY 4
#include "common.cuh"

namespace {

constexpr int TILE = 128;       // keys per tile = threads per block
constexpr int MAX_R = 4;        // head dims per thread: head_dim <= 512

template <typename TQ, typename TC, typename TO>
__global__ void __launch_bounds__(TILE)
attention_simt_kernel(const TQ* __restrict__ q, const TC* __restrict__ k_pages, const TC* __restrict__ v_pages,
                      TO* __restrict__ out, const int* __restrict__ token_seq, const int* __restrict__ token_pos,
                      const int* __restrict__ table, int table_stride, int nh, int nkv, int hd, int hdv, int ldv, float scale,
                      float softcap, int window, int keep, int sink, const float* __restrict__ sink_v, const float* __restrict__ key_scales,
                      const float* __restrict__ slopes, int page_size, int n_pages, int* status) {
    ik_pdl_wait();
    ik_pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char smem[];
    size_t* row = (size_t*)smem;              // [TILE] row of key j in the pages (page, kv head, place), times the head size = its offset
    float* qs = (float*)(row + TILE);         // [hd]
    float* sc = qs + hd;                      // [TILE]
    float* red = sc + TILE;                   // [32]

    const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int kvh = h / (nh / nkv);
    const int pos = token_pos[t], seq = token_seq[t];
    const int j0 = (window > 0 && pos + 1 > window) ? pos + 1 - window : 0;

    const TQ* qrow = q + ((size_t)t * nh + h) * hd;
    for (int i = tid; i < hd; i += TILE) qs[i] = ik_ld(qrow, i);

    // the sink stands at the head of the running softmax: a maximum of 0 whose weight exp(0 - 0) = 1 is already in the sum
    // (with sink_v the sink's score is the head's own number instead of 0; it is not scaled)
    float m = sink ? (sink_v ? sink_v[h] : 0.f) : -INFINITY, l = sink ? 1.f : 0.f, o[MAX_R];
    #pragma unroll
    for (int r = 0; r < MAX_R; r++) o[r] = 0.f;
    __syncthreads();

    // every tile visited holds at least one visible key
    const int kept_tiles = (keep + TILE - 1) / TILE;
    for (int tile = keep > 0 ? 0 : j0 / TILE; tile * TILE <= pos; tile = tile + 1 >= kept_tiles ? max(tile + 1, j0 / TILE) : tile + 1) {
        const int base = tile * TILE, j = base + tid;
        const bool valid = (j >= j0 || j < keep) && j <= pos;
        float s = -INFINITY;
        size_t off = 0;
        if (valid) {
            const int page = table[(size_t)seq * table_stride + j / page_size];
            if (page < 0 || page >= n_pages) {
                ik_set_status(status, IK_STATUS_READ_NO_PAGE);
                off = 0;
            } else {
                off = ((size_t)page * nkv + kvh) * page_size + (j % page_size);
            }
            const TC* kr = k_pages + off * hd;
            float dot = 0.f;
            for (int i = 0; i < hd; i++) dot = fmaf(qs[i], ik_ld(kr, i), dot);
            s = dot * scale;
            if (key_scales) s *= key_scales[off];
            if (softcap > 0.f) s = softcap * tanhf(s / softcap);
            if (slopes) s = fmaf(-slopes[h], (float)(pos - j), s);
        }
        row[tid] = off;
        const float tile_max = ik_block_max<TILE>(s, red);
        const float m_new = fmaxf(m, tile_max);
        const float p = valid ? expf(s - m_new) : 0.f;
        sc[tid] = p;
        const float tile_sum = ik_block_sum<TILE>(p, red);     // its barriers also publish sc[] and row[]
        const float alpha = expf(m - m_new);                   // 0 on the first tile (m = -inf)
        l = l * alpha + tile_sum;
        const int n_in_tile = min(TILE, pos - base + 1);
        #pragma unroll
        for (int r = 0; r < MAX_R; r++) {
            const int i = tid + r * TILE;
            if (i < hdv) {
                float acc = o[r] * alpha;
                for (int jj = 0; jj < n_in_tile; jj++) {
                    const float pj = sc[jj];
                    if (pj != 0.f) acc = fmaf(pj, ik_ld(v_pages + row[jj] * ldv, i), acc);
                }
                o[r] = acc;
            }
        }
        m = m_new;
        __syncthreads();                                       // sc[] and row[] are rewritten by the next tile
    }
    TO* orow = out + ((size_t)t * nh + h) * hdv;
    const float inv = 1.0f / l;
    #pragma unroll
    for (int r = 0; r < MAX_R; r++) {
        const int i = tid + r * TILE;
        if (i < hdv) ik_st(orow, i, o[r] * inv);
    }
}

}  // namespace

IK_EXPORT int ik_attention_simt(const void* q, int q_dtype, const void* k_pages, const void* v_pages, int cache_dtype,
                                void* out, int out_dtype, const int* token_seq, const int* token_pos, const int* table,
                                int table_stride, int T, int nh, int nkv, int hd, int hdv, int ldv, float scale, float softcap, int window, int keep,
                                int sink, const float* sink_v, const float* key_scales, const float* slopes, int page_size, int n_pages, int* status,
                                cudaStream_t stream) {
    if (ldv < hdv) return IK_BAD_ARGUMENT;
    if (T < 0 || nh <= 0 || nkv <= 0 || nh % nkv || hd <= 0 || hdv <= 0 || hdv > TILE * MAX_R || page_size <= 0 || softcap < 0.f || keep < 0) return IK_BAD_ARGUMENT;
    if (q_dtype != out_dtype) return IK_BAD_ARGUMENT;
    if (T == 0) return IK_OK;
    dim3 grid(T, nh);
    const size_t smem = (size_t)(hd + TILE + 32) * sizeof(float) + TILE * sizeof(size_t);
#define IK_ATT(TQ, TC)                                                                                                \
    IK_RETURN_IF_ERROR(ik_launch(attention_simt_kernel<TQ, TC, TQ>, grid, TILE, smem, stream, (const TQ*)q, (const TC*)k_pages, (const TC*)v_pages, \
        (TQ*)out, token_seq, token_pos, table, table_stride, nh, nkv, hd, hdv, ldv, scale, softcap, window, keep, sink, sink_v, key_scales, slopes, page_size, n_pages, status))
    if (q_dtype == IK_F32 && cache_dtype == IK_F32) IK_ATT(float, float);
    else if (q_dtype == IK_BF16 && cache_dtype == IK_BF16) IK_ATT(__nv_bfloat16, __nv_bfloat16);
    else if (q_dtype == IK_F32 && cache_dtype == IK_BF16) IK_ATT(float, __nv_bfloat16);
    else if (q_dtype == IK_BF16 && cache_dtype == IK_F32) IK_ATT(__nv_bfloat16, float);
    else return IK_BAD_ARGUMENT;
#undef IK_ATT
    IK_LAUNCH_STATUS();
}
