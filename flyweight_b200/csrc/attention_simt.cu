// Causal grouped-query attention over the paged cache, plain SIMT, fp32 arithmetic.
//
// One block per (query token, KV head).  The block walks the keys that the token may
// see, lo..pos (lo = max(0, pos-window+1) with a window, else 0; with `keep` also the
// positions below it) in tiles of 32
// positions that start at multiples of 32, stages each K and V tile in shared memory
// once, and lets its warps run an online softmax for the query heads of that KV head.
// A tile never straddles a page (the page size is a multiple of 32).  The walk and the
// reduction order depend only on the token's own position, never on how the batch was
// cut, so the result for a token is the same in a whole prompt, in a portion, or as a
// single decoded token.
//
// This kernel is the attention of the 32-bit path, and the fallback of the bfloat16
// path for head sizes or group sizes the tensor-core kernels refuse.
#include "common.cuh"

using namespace fwb;

namespace {

constexpr int WARPS = 4;
constexpr int TILE = 32;
constexpr int MAX_HPW = 4;   // query heads per warp  -> 16 heads of a group per block (larger groups: more blocks)
constexpr int MAX_DPL = 8;   // head channels per lane -> head size <= 256

template <typename TQ, typename TC, typename TO>
__global__ void __launch_bounds__(WARPS * 32)
attention_simt_kernel(const TQ* __restrict__ q, const TC* __restrict__ k_pool,
                      const TC* __restrict__ v_pool, const int* __restrict__ positions,
                      const int* __restrict__ tok_seg, const int* __restrict__ block_table,
                      int max_pages, int page_size, TO* __restrict__ out, int nh, int nkv, int hd,
                      int window, float scale, const float* __restrict__ sink, float softcap, int keep) {
    fwb::pdl_entry();
    extern __shared__ float smem[];
    const int group = nh / nkv;
    // a block takes up to WARPS * MAX_HPW query heads of its KV head; a larger group is cut over blockIdx.z
    const int g0 = blockIdx.z * (WARPS * MAX_HPW);
    const int mine = group - g0 < WARPS * MAX_HPW ? group - g0 : WARPS * MAX_HPW;
    float* qs = smem;                         // [mine][hd]
    float* ks = qs + mine * hd;               // [TILE][hd+1]
    float* vs = ks + TILE * (hd + 1);         // [TILE][hd]
    const int t = blockIdx.x, kvh = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pos = positions[t];
    const int* table = block_table + (size_t)tok_seg[t] * max_pages;
    const int lo = fwb::first_visible_key(pos, window);

    for (int i = threadIdx.x; i < mine * hd; i += blockDim.x)
        qs[i] = to_f32<TQ>(q[((size_t)t * nh + (size_t)kvh * group + g0) * hd + i]);

    float m[MAX_HPW], l[MAX_HPW], acc[MAX_HPW][MAX_DPL];
#pragma unroll
    for (int a = 0; a < MAX_HPW; ++a) {
        // a sink: a key of score sink[head] (not scaled, not capped) whose value is zero starts the row
        const int g = warp + a * WARPS;
        const bool sunk = sink != nullptr && g < mine;
        m[a] = sunk ? sink[kvh * group + g0 + g] : -INFINITY;
        l[a] = sunk ? 1.0f : 0.0f;
#pragma unroll
        for (int d = 0; d < MAX_DPL; ++d) acc[a][d] = 0.0f;
    }
    const float inv_cap = softcap > 0.0f ? 1.0f / softcap : 0.0f;

    const KeyTiles walk = fwb::key_tiles(lo, pos, keep, TILE);
    for (int tile = 0; tile < walk.count; ++tile) {
        const int base = walk.at(tile) * TILE;
        __syncthreads();
        const int page = table[base / page_size];
        const size_t src = (((size_t)page * nkv + kvh) * page_size + (base % page_size)) * hd;
        const int valid = pos - base + 1 < TILE ? pos - base + 1 : TILE;   // rows of the tile in use
        for (int i = threadIdx.x; i < TILE * hd; i += blockDim.x) {
            const int r = i / hd, c = i - r * hd;
            const bool live = r < valid;
            ks[r * (hd + 1) + c] = live ? to_f32<TC>(k_pool[src + i]) : 0.0f;
            vs[i] = live ? to_f32<TC>(v_pool[src + i]) : 0.0f;
        }
        __syncthreads();
        const int kpos = base + lane;
        const bool seen = (kpos >= lo || kpos < keep) && kpos <= pos;
#pragma unroll
        for (int a = 0; a < MAX_HPW; ++a) {
            const int g = warp + a * WARPS;
            if (g >= mine) break;
            const float* qh = qs + g * hd;
            const float* kr = ks + lane * (hd + 1);
            float s = 0.0f;
            for (int d = 0; d < hd; ++d) s = fmaf(qh[d], kr[d], s);
            s *= scale;
            if (softcap > 0.0f) s = softcap * tanhf(s * inv_cap);
            s = seen ? s : -INFINITY;
            const float tile_max = warp_max(s);
            if (tile_max == -INFINITY) continue;   // nothing visible in this tile (warp-uniform)
            const float m_new = fmaxf(m[a], tile_max);
            const float p = seen ? expf(s - m_new) : 0.0f;
            const float corr = expf(m[a] - m_new);  // m[a] == -inf gives 0
            l[a] = l[a] * corr + warp_sum(p);
            m[a] = m_new;
#pragma unroll
            for (int d = 0; d < MAX_DPL; ++d) acc[a][d] *= corr;
            for (int j = 0; j < valid; ++j) {
                const float pj = __shfl_sync(0xffffffffu, p, j);
#pragma unroll
                for (int d = 0; d < MAX_DPL; ++d) {
                    const int c = lane + 32 * d;
                    if (c < hd) acc[a][d] = fmaf(pj, vs[j * hd + c], acc[a][d]);
                }
            }
        }
    }
#pragma unroll
    for (int a = 0; a < MAX_HPW; ++a) {
        const int g = warp + a * WARPS;
        if (g >= mine) break;
        const float inv = 1.0f / l[a];
        TO* dst = out + ((size_t)t * nh + (size_t)kvh * group + g0 + g) * hd;
#pragma unroll
        for (int d = 0; d < MAX_DPL; ++d) {
            const int c = lane + 32 * d;
            if (c < hd) dst[c] = from_f32<TO>(acc[a][d] * inv);
        }
    }
}

}  // namespace

// q, out: [T][nh*hd].  k_pool, v_pool: [pages][nkv][page_size][hd].  positions, tok_seg: [T].
// block_table: [S][max_pages].  The keys of every position <= a token's own must
// already be in the cache (this step's included).  Dtype flags: 0 fp32, 1 bf16.
FWB_API int fwb_attention_simt(const void* q, int q_bf16, const void* k_pool, const void* v_pool,
                               int cache_bf16, const int* positions, const int* tok_seg,
                               const int* block_table, int max_pages, int page_size, void* out,
                               int out_bf16, int T, int nh, int nkv, int hd, int window, float scale,
                               cudaStream_t stream);

// The general form.  sink: fp32 [nh] or null -- a score per head (not scaled, not capped) that joins the
// row's softmax denominator and has no value.  softcap > 0: score <- softcap * tanh(score / softcap)
// behind the scale.  keep > 0 (with a sliding window): the sequence's first `keep` positions stay visible
// however far the window has moved on.
FWB_API int fwb_attention_simt_sink(const void* q, int q_bf16, const void* k_pool, const void* v_pool,
                                    int cache_bf16, const int* positions, const int* tok_seg,
                                    const int* block_table, int max_pages, int page_size, void* out,
                                    int out_bf16, int T, int nh, int nkv, int hd, int window, float scale,
                                    const float* sink, float softcap, int keep, cudaStream_t stream) {
    if (T <= 0) return FWB_OK;
    if (keep < 0 || (keep > 0 && window <= 0)) return FWB_BAD_ARGUMENT;
    if (!q || !k_pool || !v_pool || !positions || !tok_seg || !block_table || !out)
        return FWB_BAD_ARGUMENT;
    if (nh <= 0 || nkv <= 0 || nh % nkv != 0 || hd <= 0 || max_pages <= 0) return FWB_BAD_ARGUMENT;
    if (page_size <= 0 || page_size % TILE != 0) return FWB_UNSUPPORTED;
    const int group = nh / nkv;
    const int cuts = (group + WARPS * MAX_HPW - 1) / (WARPS * MAX_HPW);
    if (hd > 32 * MAX_DPL || nkv > 65535 || cuts > 65535) return FWB_UNSUPPORTED;
    const size_t smem = ((size_t)(cuts > 1 ? WARPS * MAX_HPW : group) * hd + (size_t)TILE * (2 * hd + 1)) * sizeof(float);
    using bf = __nv_bfloat16;
    dim3 grid(T, nkv, cuts);
#define FWB_ATTN(TQ, TC, TO)                                                                      \
    do {                                                                                          \
        auto kernel = attention_simt_kernel<TQ, TC, TO>;                                          \
        if (smem > 48 * 1024) {                                                                   \
            cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                                 (int)smem);                                      \
            if (e != cudaSuccess) return (int)e;                                                  \
        }                                                                                         \
        fwb::pdl(kernel, grid, WARPS * 32, smem, stream)((const TQ*)q, (const TC*)k_pool,               \
                                                   (const TC*)v_pool, positions, tok_seg,         \
                                                   block_table, max_pages, page_size, (TO*)out,   \
                                                   nh, nkv, hd, window, scale, sink, softcap, keep); \
    } while (0)
    if (!q_bf16 && !cache_bf16 && !out_bf16) FWB_ATTN(float, float, float);
    else if (q_bf16 && cache_bf16 && out_bf16) FWB_ATTN(bf, bf, bf);
    else return FWB_UNSUPPORTED;
#undef FWB_ATTN
    return fwb_launch_status();
}

FWB_API int fwb_attention_simt(const void* q, int q_bf16, const void* k_pool, const void* v_pool,
                               int cache_bf16, const int* positions, const int* tok_seg,
                               const int* block_table, int max_pages, int page_size, void* out,
                               int out_bf16, int T, int nh, int nkv, int hd, int window, float scale,
                               cudaStream_t stream) {
    return fwb_attention_simt_sink(q, q_bf16, k_pool, v_pool, cache_bf16, positions, tok_seg, block_table,
                                   max_pages, page_size, out, out_bf16, T, nh, nkv, hd, window, scale, nullptr,
                                   0.0f, 0, stream);
}
