// Attention over a cached low-rank latent for bfloat16 rows of any length up to 576 entries.
//
// A cache row is [ latent (rank) | turned key part (rot) | 0 ], `row` entries.  Three kernels:
//
//   fwb_latent_attention_mma   every query head as one row of the cache row's layout (a query carried into the
//                      latent's space), against the cached rows themselves; values are a row's first `rank` columns.
//                      mma.sync m16n8k16, fp32 accumulation and softmax.  One CTA takes 16 or 32 query rows (heads
//                      of one token, or of a few neighbouring tokens) and one slice of the context, 64 keys at a
//                      time: a cached row is read once for all of them.  Eight or sixteen warps share a tile's
//                      scores (16 rows by 8 or 16 keys each, the queries in registers), the scores meet in shared
//                      memory for the online softmax, and for the weighted sum every warp owns a share of the
//                      latent's columns.
//                      Slices are merged by a second kernel through fp32 scratch.  Steps of single tokens, and
//                      prompts whose heads fit no prompt kernel.
//   fwb_latent_gather  the cached rows that the prompts of a step may see, side by side and padded to runs of 64
//                      (the input of a product that expands them into head keys and head values)
//   fwb_latent_spread  queries with their rotated part turned, laid out for heads of `hd` channels
//
// Key tiles start at multiples of 64 and are visited in ascending order, whatever the cut.
#include "common.cuh"

using namespace fwb;

namespace {

constexpr int KEYS = 64;               // keys per tile == page size
constexpr int PAD = 8;                 // bf16 entries behind a shared row (rows then start 4 banks apart)
constexpr int PS = KEYS + 8;           // bf16 entries of a row of probabilities
constexpr int SS = KEYS + 4;           // fp32 entries of a row of scores
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
    const uint32_t s = static_cast<uint32_t>(__cvta_generic_to_shared(smem));
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
    asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const __nv_bfloat16* row) {
    const uint32_t at = (uint32_t)__cvta_generic_to_shared(row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const __nv_bfloat16* row) {
    const uint32_t at = (uint32_t)__cvta_generic_to_shared(row);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct RowsParams {
    const __nv_bfloat16* qa;     // [T][heads][row]
    const __nv_bfloat16* pool;   // [pages][64][row]
    const float* sink;           // [heads] or null: a score per head that joins the softmax without a value
    const int* positions;        // [T]
    const int* tok_seg;          // [T] (single tokens)
    const int* seg_start;        // [S + 1] (tiles of prompts)
    const int* tile_seg;         // [tiles] or null: blockIdx.x is a token
    const int* tile_tok0;
    const int* block_table;      // [S][max_pages]
    __nv_bfloat16* out;          // [T][heads][rank]
    float* part_o;               // [T][heads][splits][rank], not normalised (splits > 1)
    float* part_ml;              // [T][heads][splits][2]
    int max_pages, heads, heads_per_cta, tokens_per_tile, rank, row, splits, tiles_per_split, stages;
    float scale_log2;
};

// MT: bands of 16 query rows.  KS: the most 16-entry steps of a row (steps behind a shorter row's last repeat it
// against zero queries: no branch in the loop).  NB: 16-column blocks of the latent a warp owns.
template <int MT, int KS, int NB, int WARPS>
__global__ void __launch_bounds__(WARPS * 32, WARPS == 8 && KS <= 18 && MT == 1 ? 2 : 1)
latent_rows_kernel(const RowsParams prm) {
    fwb::pdl_entry();
    constexpr int THREADS = WARPS * 32, M = MT * 16;
    constexpr int NT = MT * 8 / WARPS, OWN = M / WARPS;     // 8-key tiles of a warp's scores; rows of its softmax
    constexpr int STEPS = KS * 16;
    constexpr int LPR = 32 / OWN, PER = KEYS / LPR;         // lanes of a row's softmax, scores a lane
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const int row = prm.row, RS = row + PAD, rank = prm.rank;
    __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(smem_raw);             // [stages][KEYS][RS]
    __nv_bfloat16* Ps = Ks + (size_t)prm.stages * KEYS * RS;                    // [M][PS]
    float* Sc = reinterpret_cast<float*>(Ps + M * PS);                          // [M][SS]
    float* corr_s = Sc + M * SS;                                                // [M]
    float* l_s = corr_s + M;                                                    // [M]
    float* m_s = l_s + M;                                                       // [M]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;

    int seg, tok0, n_tok = 1;
    const int h0 = blockIdx.y * prm.heads_per_cta, split = blockIdx.z;
    const int nh = prm.heads - h0 < prm.heads_per_cta ? prm.heads - h0 : prm.heads_per_cta;
    if (prm.tile_seg) {
        const int item = gridDim.x - 1 - blockIdx.x;        // a prompt's last tiles walk the most keys: they go first
        seg = prm.tile_seg[item];
        tok0 = prm.tile_tok0[item];
        n_tok = prm.seg_start[seg + 1] - tok0;
        if (n_tok > prm.tokens_per_tile) n_tok = prm.tokens_per_tile;
    } else {
        tok0 = blockIdx.x;
        seg = prm.tok_seg[tok0];
    }
    const int rows = n_tok * nh;
    const int pos_last = prm.positions[tok0 + n_tok - 1];
    const int* table = prm.block_table + (size_t)seg * prm.max_pages;
    const int n_tiles = pos_last / KEYS + 1;
    const int first = split * prm.tiles_per_split;
    const int last = first + prm.tiles_per_split < n_tiles ? first + prm.tiles_per_split : n_tiles;
    auto row_at = [&](int r, size_t& at) {                  // entry (token, head) of row r; false: no such row
        if (r >= rows) return false;
        at = (size_t)(tok0 + r / nh) * prm.heads + h0 + r % nh;
        return true;
    };

    // this warp's part of the scores: 16 rows by NT * 8 keys
    const int mt0 = MT == 2 ? (warp & 1) : 0, key0 = (MT == 2 ? (warp >> 1) : warp) * NT * 8;
    static_assert(NT == 1 || NT == 2, "a warp scores 8 or 16 keys of a tile");
    uint32_t qf[KS][4];
    {
        size_t lo = 0, hi = 0;
        const bool has_lo = row_at(mt0 * 16 + g, lo), has_hi = row_at(mt0 * 16 + g + 8, hi);
        const __nv_bfloat16* q_lo = prm.qa + lo * row;
        const __nv_bfloat16* q_hi = prm.qa + hi * row;
#pragma unroll
        for (int k = 0; k < KS; ++k) {
            const int d = k * 16 + 2 * t;
            const bool in = k * 16 < row;
            qf[k][0] = in && has_lo ? *reinterpret_cast<const uint32_t*>(q_lo + d) : 0u;
            qf[k][1] = in && has_hi ? *reinterpret_cast<const uint32_t*>(q_hi + d) : 0u;
            qf[k][2] = in && has_lo ? *reinterpret_cast<const uint32_t*>(q_lo + d + 8) : 0u;
            qf[k][3] = in && has_hi ? *reinterpret_cast<const uint32_t*>(q_hi + d + 8) : 0u;
        }
    }
    // this lane's row of the softmax (LPR lanes share one): running maximum, a lane's share of the running sum, last
    // visible key
    const int own = warp * OWN + lane / LPR, sub = lane % LPR;
    float m_run = -INFINITY, l_run = 0.0f;
    int hi_key = -1;
    if (own < rows) {
        hi_key = prm.positions[tok0 + own / nh];
        if (prm.sink && split == 0) {
            m_run = prm.sink[h0 + own % nh] * LOG2E;
            l_run = sub == 0 ? 1.0f : 0.0f;
        }
    }
    float acc[MT][NB][2][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nb = 0; nb < NB; ++nb)
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[mt][nb][j >> 2][j & 3] = 0.0f;

    const int chunks = row >> 3, row_step = THREADS / chunks, chunk_step = THREADS % chunks;
    const int row_first = threadIdx.x / chunks, chunk_first = threadIdx.x % chunks;
    auto issue = [&](int tile) {
        if (tile < last) {
            __nv_bfloat16* dst = Ks + (size_t)((tile - first) % prm.stages) * KEYS * RS;
            const __nv_bfloat16* src = prm.pool + (size_t)table[tile] * KEYS * row;
            const int seen = pos_last - tile * KEYS + 1;    // rows behind the last visible key are zero
            for (int r = row_first, c = chunk_first; r < KEYS;) {
                if (r < seen) cp_async16(dst + r * RS + c * 8, src + r * row + c * 8);
                else *reinterpret_cast<uint4*>(dst + r * RS + c * 8) = make_uint4(0u, 0u, 0u, 0u);
                r += row_step;
                c += chunk_step;
                if (c >= chunks) {
                    c -= chunks;
                    ++r;
                }
            }
        }
        cp_async_commit();
    };
    for (int s = 0; s < prm.stages - 1; ++s) issue(first + s);
    for (int tile = first; tile < last; ++tile) {
        if (prm.stages == 2) cp_async_wait<0>();
        else cp_async_wait<1>();
        __syncthreads();                                    // the tile is in place; everybody is done with the one before
        issue(tile + prm.stages - 1);
        const __nv_bfloat16* kt = Ks + (size_t)((tile - first) % prm.stages) * KEYS * RS;
        {
            float s[2][NT][4];
#pragma unroll
            for (int j = 0; j < 2 * NT * 4; ++j) s[j / (NT * 4)][(j >> 2) % NT][j & 3] = 0.0f;
            if (NT == 2) {
                const __nv_bfloat16* kb = kt + (key0 + (lane & 7) + ((lane >> 4) << 3)) * RS + (((lane >> 3) & 1) << 3);
#pragma unroll
                for (int k = 0; k < KS; ++k) {
                    uint32_t b[4];
                    ldsm4(b, kb + (STEPS == row || k * 16 < row ? k * 16 : row - 16));
                    mma_bf16(s[k & 1][0], qf[k], b[0], b[1]);
                    mma_bf16(s[k & 1][NT - 1], qf[k], b[2], b[3]);
                }
            } else {
                // 8 keys by two steps at a time
                const __nv_bfloat16* kb = kt + (key0 + (lane & 7)) * RS;
                const int at = (lane >> 3) << 3;
#pragma unroll
                for (int k = 0; k < KS; k += 2) {
                    uint32_t b[4];
                    const int c = k * 16 + at;
                    ldsm4(b, kb + (c < row ? c : row - 8));
                    mma_bf16(s[0][0], qf[k], b[0], b[1]);
                    mma_bf16(s[1][0], qf[k + 1], b[2], b[3]);
                }
            }
#pragma unroll
            for (int nt = 0; nt < NT; ++nt)
#pragma unroll
                for (int half = 0; half < 2; ++half)
                    *reinterpret_cast<float2*>(Sc + (mt0 * 16 + g + 8 * half) * SS + key0 + nt * 8 + 2 * t) =
                        make_float2(s[0][nt][2 * half] + s[1][nt][2 * half], s[0][nt][2 * half + 1] + s[1][nt][2 * half + 1]);
        }
        __syncthreads();
        {
            // groups of four neighbouring keys, LPR groups apart
            float v[PER];
            float top = -INFINITY;
#pragma unroll
            for (int j = 0; j < PER; j += 4) {
                const int c = 4 * (sub + (j / 4) * LPR);
                const float4 s4 = *reinterpret_cast<const float4*>(Sc + own * SS + c);
                const int left = hi_key - (tile * KEYS + c);                // visible: key c + i with i <= left
                v[j] = left >= 0 ? s4.x * prm.scale_log2 : -INFINITY;
                v[j + 1] = left >= 1 ? s4.y * prm.scale_log2 : -INFINITY;
                v[j + 2] = left >= 2 ? s4.z * prm.scale_log2 : -INFINITY;
                v[j + 3] = left >= 3 ? s4.w * prm.scale_log2 : -INFINITY;
                top = fmaxf(fmaxf(top, fmaxf(v[j], v[j + 1])), fmaxf(v[j + 2], v[j + 3]));
            }
#pragma unroll
            for (int step = LPR / 2; step > 0; step >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, step));
            const float m_new = fmaxf(m_run, top);
            const float base = m_new == -INFINITY ? 0.0f : m_new;           // a row that has seen no key yet
            const float corr = exp2f(m_run - base);
            float sum = 0.0f;
#pragma unroll
            for (int j = 0; j < PER; j += 4) {
                const float p0 = exp2f(v[j] - base), p1 = exp2f(v[j + 1] - base);
                const float p2 = exp2f(v[j + 2] - base), p3 = exp2f(v[j + 3] - base);
                sum += (p0 + p1) + (p2 + p3);
                const __nv_bfloat162 lo = __floats2bfloat162_rn(p0, p1), hi = __floats2bfloat162_rn(p2, p3);
                *reinterpret_cast<uint2*>(Ps + own * PS + 4 * (sub + (j / 4) * LPR)) =
                    make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
            }
            l_run = fmaf(l_run, corr, sum);
            m_run = m_new;
            if (sub == 0) corr_s[own] = corr;
        }
        __syncthreads();
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
            const float up = corr_s[mt * 16 + g], down = corr_s[mt * 16 + g + 8];
#pragma unroll
            for (int nb = 0; nb < NB; ++nb)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    acc[mt][nb][h][0] *= up;
                    acc[mt][nb][h][1] *= up;
                    acc[mt][nb][h][2] *= down;
                    acc[mt][nb][h][3] *= down;
                }
        }
#pragma unroll
        for (int kk = 0; kk < KEYS / 16; ++kk) {
            uint32_t p[MT][4];
#pragma unroll
            for (int mt = 0; mt < MT; ++mt)
                ldsm4(p[mt], Ps + (mt * 16 + (lane & 15)) * PS + kk * 16 + ((lane >> 4) << 3));
#pragma unroll
            for (int nb = 0; nb < NB; ++nb) {
                // (a block behind the last column repeats that one; nobody stores its sums)
                const int col = (warp + WARPS * nb) * 16 < row ? (warp + WARPS * nb) * 16 : row - 16;
                uint32_t b[4];
                ldsm4t(b, kt + (kk * 16 + (lane & 15)) * RS + col + ((lane >> 4) << 3));
#pragma unroll
                for (int mt = 0; mt < MT; ++mt) {
                    mma_bf16(acc[mt][nb][0], p[mt], b[0], b[1]);
                    mma_bf16(acc[mt][nb][1], p[mt], b[2], b[3]);
                }
            }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int step = LPR / 2; step > 0; step >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, step);
    if (sub == 0) {
        l_s[own] = l_run;
        m_s[own] = m_run;
    }
    __syncthreads();
    const bool whole = prm.splits == 1;
    for (int r = threadIdx.x; !whole && r < rows; r += THREADS) {
        size_t at = 0;
        row_at(r, at);
        float* ml = prm.part_ml + (at * prm.splits + split) * 2;
        ml[0] = m_s[r];
        ml[1] = l_s[r];
    }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int r = mt * 16 + g + 8 * half;
            size_t at = 0;
            if (!row_at(r, at)) continue;
            const float inv = whole ? 1.0f / l_s[r] : 1.0f;
            if (!whole && m_s[r] == -INFINITY) continue;     // (a slice without a visible key: the merge skips it)
#pragma unroll
            for (int nb = 0; nb < NB; ++nb)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const int c = (warp + WARPS * nb) * 16 + h * 8 + 2 * t;
                    const float v0 = acc[mt][nb][h][2 * half] * inv, v1 = acc[mt][nb][h][2 * half + 1] * inv;
                    if (whole) {
                        if (c < rank) prm.out[at * rank + c] = __float2bfloat16_rn(v0);
                        if (c + 1 < rank) prm.out[at * rank + c + 1] = __float2bfloat16_rn(v1);
                    } else {
                        float* dst = prm.part_o + (at * prm.splits + split) * rank + c;
                        if (c < rank) dst[0] = v0;
                        if (c + 1 < rank) dst[1] = v1;
                    }
                }
        }
}

// One block per (token, head): the slices' partial results by the usual rule.
__global__ void __launch_bounds__(128)
latent_rows_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                         __nv_bfloat16* __restrict__ out, int splits, int rank) {
    fwb::pdl_entry();
    const size_t at = blockIdx.x;
    const float* ml = part_ml + at * splits * 2;
    float m = -INFINITY, l = 0.0f;
    for (int s = 0; s < splits; ++s) m = fmaxf(m, ml[2 * s]);
    for (int s = 0; s < splits; ++s) l += ml[2 * s] == -INFINITY ? 0.0f : exp2f(ml[2 * s] - m) * ml[2 * s + 1];
    const float inv = 1.0f / l;
    for (int c = threadIdx.x; c < rank; c += blockDim.x) {
        float v = 0.0f;
        for (int s = 0; s < splits; ++s)
            if (ml[2 * s] != -INFINITY) v = fmaf(exp2f(ml[2 * s] - m), part_o[(at * splits + s) * rank + c], v);
        out[at * rank + c] = __float2bfloat16_rn(v * inv);
    }
}

// One block per run of 64 rows: `out` [n_pages][64][row] receives logical page page_no[i] of segment page_seg[i];
// rows behind the segment's last token are zero.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ pool, const int* __restrict__ page_seg, const int* __restrict__ page_no,
                     const int* __restrict__ block_table, int max_pages, const int* __restrict__ seg_start,
                     const int* __restrict__ seg_pos0, uint4* __restrict__ out, int chunks) {
    fwb::pdl_entry();
    const int i = blockIdx.x, seg = page_seg[i], no = page_no[i];
    const int seen = seg_pos0[seg] + seg_start[seg + 1] - seg_start[seg] - no * KEYS;
    const uint4* src = pool + (size_t)block_table[(size_t)seg * max_pages + no] * KEYS * chunks;
    uint4* dst = out + (size_t)i * KEYS * chunks;
    const int live = (seen < KEYS ? seen : KEYS) * chunks;
    for (int j = threadIdx.x; j < KEYS * chunks; j += blockDim.x) dst[j] = j < live ? src[j] : make_uint4(0u, 0u, 0u, 0u);
}

// One block per token: q [T][heads][dim + rot] -> out [T][heads][hd] with the rotated part turned by the token's
// position and zeros behind it.  Two neighbouring channels a thread and turn (dim, rot, hd even).
__global__ void __launch_bounds__(256)
latent_spread_kernel(const __nv_bfloat16* __restrict__ q, const float* __restrict__ table,
                     const int* __restrict__ positions, __nv_bfloat16* __restrict__ out, int heads, int dim, int rot,
                     int rot_dims, int interleaved, int hd) {
    fwb::pdl_entry();
    const int t = blockIdx.x, half = rot_dims >> 1, width = dim + rot, pairs = hd >> 1;
    const float* cs = table + (size_t)positions[t] * (half > 0 ? half : 1) * 2;
    for (int i = threadIdx.x; i < heads * pairs; i += blockDim.x) {
        const int h = i / pairs, c = (i - h * pairs) << 1;
        const __nv_bfloat16* src = q + ((size_t)t * heads + h) * width;
        __nv_bfloat162 v = __floats2bfloat162_rn(0.0f, 0.0f);
        if (c < width) {
            v = *reinterpret_cast<const __nv_bfloat162*>(src + c);
            const int r = c - dim;
            if (r >= 0 && r < rot_dims) {
                float a[2] = {__low2float(v), __high2float(v)};
                float o[2];
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const int k = r + j;
                    if (k >= rot_dims) {
                        o[j] = a[j];
                        continue;
                    }
                    const int pair = interleaved ? k >> 1 : (k < half ? k : k - half);
                    const int partner = interleaved ? k ^ 1 : (k < half ? k + half : k - half);
                    const float sign = (interleaved ? (k & 1) == 0 : k < half) ? -1.0f : 1.0f;
                    const float b = interleaved ? a[j ^ 1] : __bfloat162float(src[dim + partner]);
                    o[j] = a[j] * cs[2 * pair] + sign * b * cs[2 * pair + 1];
                }
                v = __floats2bfloat162_rn(o[0], o[1]);
            }
        }
        *reinterpret_cast<__nv_bfloat162*>(out + ((size_t)t * heads + h) * hd + c) = v;
    }
}

size_t rows_smem(int mt, int row, int stages) {
    const size_t m = 16 * mt;
    return (size_t)stages * KEYS * (row + PAD) * 2 + m * PS * 2 + m * SS * 4 + 3 * m * 4;
}

template <int MT, int KS, int NB, int WARPS>
int launch_rows(RowsParams prm, int items, int groups, cudaStream_t stream) {
    constexpr size_t LIMIT = WARPS == 8 && KS <= 18 && MT == 1 ? 112 * 1024 : 224 * 1024;
    prm.stages = rows_smem(MT, prm.row, 3) <= LIMIT ? 3 : 2;
    const size_t smem = rows_smem(MT, prm.row, prm.stages);
    auto kernel = latent_rows_kernel<MT, KS, NB, WARPS>;
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    fwb::pdl(kernel, dim3(items, groups, prm.splits), WARPS * 32, smem, stream)(prm);
    return fwb_launch_status();
}

}  // namespace

// Shapes the tensor-core kernel takes: rows of a multiple of 16 entries up to 576, latents up to 512.
FWB_API int fwb_latent_attention_mma_accepts(int rank, int row, int page_size) {
    return page_size == KEYS && row % 16 == 0 && row >= 16 && row <= 576 && rank > 0 && rank <= 512 && rank <= row
           && (row > 320 || rank <= 320) && (row > 192 || rank <= 192);
}

// qa: [T][heads][row] bf16; pool: [pages][64][row] bf16; out: [T][heads][rank] bf16.  With tile_seg (prompts): n_items
// tiles of up to tokens_per_tile tokens of one segment each, tokens_per_tile * heads_per_cta <= 32, splits == 1;
// without: the first n_items tokens of the step, the context cut into `splits` slices of tiles_per_split tiles (their
// partial results: part_o [n_items][heads][splits][rank], part_ml [n_items][heads][splits][2]).  heads_per_cta <= 32.
FWB_API int fwb_latent_attention_mma(const void* qa, const void* pool, const float* sink, const int* positions,
                                     const int* tok_seg, const int* seg_start, const int* tile_seg,
                                     const int* tile_tok0, const int* block_table, int max_pages, int page_size,
                                     void* out, float* part_o, float* part_ml, int n_items, int heads,
                                     int heads_per_cta, int tokens_per_tile, int rank, int row, int splits,
                                     int tiles_per_split, float scale, cudaStream_t stream) {
    if (n_items <= 0) return FWB_OK;
    if (!qa || !pool || !positions || !block_table || !out || heads <= 0 || max_pages <= 0) return FWB_BAD_ARGUMENT;
    if (tile_seg ? (!tile_tok0 || !seg_start || splits != 1) : !tok_seg) return FWB_BAD_ARGUMENT;
    if (!fwb_latent_attention_mma_accepts(rank, row, page_size)) return FWB_UNSUPPORTED;
    if (tokens_per_tile < 1 || heads_per_cta < 1 || tokens_per_tile * heads_per_cta > 32) return FWB_BAD_ARGUMENT;
    if (splits < 1 || tiles_per_split < 1 || (splits > 1 && (!part_o || !part_ml))) return FWB_BAD_ARGUMENT;
    if ((long)splits * tiles_per_split < max_pages) return FWB_BAD_ARGUMENT;
    if ((((uintptr_t)qa | (uintptr_t)pool) & 15) != 0) return FWB_UNSUPPORTED;
    const int groups = (heads + heads_per_cta - 1) / heads_per_cta;
    if (splits > 65535 || groups > 65535) return FWB_TOO_LARGE;
    RowsParams prm;
    prm.qa = static_cast<const __nv_bfloat16*>(qa);
    prm.pool = static_cast<const __nv_bfloat16*>(pool);
    prm.sink = sink;
    prm.positions = positions;
    prm.tok_seg = tok_seg;
    prm.seg_start = seg_start;
    prm.tile_seg = tile_seg;
    prm.tile_tok0 = tile_tok0;
    prm.block_table = block_table;
    prm.out = static_cast<__nv_bfloat16*>(out);
    prm.part_o = part_o;
    prm.part_ml = part_ml;
    prm.max_pages = max_pages;
    prm.heads = heads;
    prm.heads_per_cta = heads_per_cta;
    prm.tokens_per_tile = tile_seg ? tokens_per_tile : 1;
    prm.rank = rank;
    prm.row = row;
    prm.splits = splits;
    prm.tiles_per_split = tiles_per_split;
    prm.stages = 2;
    prm.scale_log2 = scale * LOG2E;
    const bool two = heads_per_cta * prm.tokens_per_tile > 16;
    int status;
    if (row <= 192)
        status = two ? launch_rows<2, 12, 1, 16>(prm, n_items, groups, stream) : launch_rows<1, 12, 2, 8>(prm, n_items, groups, stream);
    else if (row <= 288 && rank <= 256)
        status = two ? launch_rows<2, 18, 1, 16>(prm, n_items, groups, stream) : launch_rows<1, 18, 2, 8>(prm, n_items, groups, stream);
    else if (row <= 320)
        status = two ? launch_rows<2, 20, 3, 8>(prm, n_items, groups, stream) : launch_rows<1, 20, 3, 8>(prm, n_items, groups, stream);
    else
        status = two ? launch_rows<2, 36, 4, 8>(prm, n_items, groups, stream) : launch_rows<1, 36, 4, 8>(prm, n_items, groups, stream);
    if (status != FWB_OK || splits == 1) return status;
    fwb::pdl(latent_rows_merge_kernel, dim3((unsigned)((size_t)n_items * heads)), 128, 0, stream)(
        part_o, part_ml, static_cast<__nv_bfloat16*>(out), splits, rank);
    return fwb_launch_status();
}

// pool: [pages][64][row] bf16 (row a multiple of 8); page_seg, page_no: [n_pages]; out: [n_pages][64][row].
FWB_API int fwb_latent_gather(const void* pool, const int* page_seg, const int* page_no, const int* block_table,
                              int max_pages, const int* seg_start, const int* seg_pos0, void* out, int n_pages, int row,
                              cudaStream_t stream) {
    if (n_pages <= 0) return FWB_OK;
    if (!pool || !page_seg || !page_no || !block_table || !seg_start || !seg_pos0 || !out || row <= 0 || (row & 7))
        return FWB_BAD_ARGUMENT;
    fwb::pdl(latent_gather_kernel, n_pages, 256, 0, stream)((const uint4*)pool, page_seg, page_no, block_table, max_pages,
                                                            seg_start, seg_pos0, (uint4*)out, row / 8);
    return fwb_launch_status();
}

// q: [T][heads][dim + rot] bf16, out: [T][heads][hd] bf16 (dim, rot and hd even, hd >= dim + rot).
FWB_API int fwb_latent_spread(const void* q, const float* table, const int* positions, void* out, int T, int heads,
                              int dim, int rot, int rot_dims, int interleaved, int hd, cudaStream_t stream) {
    if (T <= 0) return FWB_OK;
    if (!q || !table || !positions || !out || heads <= 0 || dim < 0 || rot < 0 || rot_dims < 0 || rot_dims > rot
        || (rot_dims & 1) || hd < dim + rot)
        return FWB_BAD_ARGUMENT;
    if ((dim | rot | hd) & 1) return FWB_UNSUPPORTED;
    fwb::pdl(latent_spread_kernel, T, 256, 0, stream)((const __nv_bfloat16*)q, table, positions, (__nv_bfloat16*)out, heads,
                                                      dim, rot, rot_dims, interleaved, hd);
    return fwb_launch_status();
}
