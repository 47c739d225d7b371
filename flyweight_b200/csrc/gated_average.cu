// A gated average over time (minGRU): a recurrence with one number of state per channel and request, whose
// gates read only the current token.
//
//   z = sigmoid(p_z + b_z),   u = p_x + b_x,   candidate = u + 1/2 (u >= 0) | sigmoid(u) (u < 0)
//   S_t = (1 - z) S_(t-1) + z candidate,       out_t = S_t * silu(p_g)
//
// p_z, p_x, p_g are columns of one fp32 projection row per token; gates, candidate, state and their products
// are fp32, the state lives in the request's slot.
//
//   step kernel  one token a segment (decoding): a thread owns VEC channels.
//   walk kernel  portions of prompts.  Because S_t = a_t S_(t-1) + b_t composes -- two stretches (A, B) then
//       (A', B') make (A' A, A' B + B') -- the tokens of a segment are cut over warps (8 tokens each) and over
//       the CTAs of a cluster (128 tokens each), a warp keeps its tokens' a, b and gates in registers, and the
//       stretches' (A, B) go around through shared memory and distributed shared memory.  Every projection row
//       is read once, and nothing but the output and the final state is written.  A segment longer than the
//       cluster's stretch goes on in rounds, the state in front of a round being the one behind the last.
#include <cooperative_groups.h>

#include "common.cuh"

using namespace fwb;
namespace cg = cooperative_groups;

namespace {

constexpr int WARPS = 16;
constexpr int TOKENS = 8;                     // tokens a warp
template <typename TO> constexpr bool quick() { return sizeof(TO) == 2; }
constexpr int STRETCH = WARPS * TOKENS;       // tokens a CTA and round

template <int VEC> struct Pack { float v[VEC]; };

template <int VEC>
__device__ __forceinline__ Pack<VEC> load_vec(const float* at) {
    Pack<VEC> r;
    if constexpr (VEC == 4) {
        const float4 f = *reinterpret_cast<const float4*>(at);
        r.v[0] = f.x, r.v[1] = f.y, r.v[2] = f.z, r.v[3] = f.w;
    } else if constexpr (VEC == 2) {
        const float2 f = *reinterpret_cast<const float2*>(at);
        r.v[0] = f.x, r.v[1] = f.y;
    } else {
        r.v[0] = *at;
    }
    return r;
}
template <int VEC>
__device__ __forceinline__ void store_vec(float* at, const Pack<VEC>& r) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(at) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else if constexpr (VEC == 2) *reinterpret_cast<float2*>(at) = make_float2(r.v[0], r.v[1]);
    else *at = r.v[0];
}
template <int VEC>
__device__ __forceinline__ void store_vec(__nv_bfloat16* at, const Pack<VEC>& r) {
    if constexpr (VEC == 4) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
        uint2 bits;
        bits.x = *reinterpret_cast<const uint32_t*>(&lo);
        bits.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(at) = bits;
    } else if constexpr (VEC == 2) {
        *reinterpret_cast<__nv_bfloat162*>(at) = __floats2bfloat162_rn(r.v[0], r.v[1]);
    } else {
        *at = __float2bfloat16_rn(r.v[0]);
    }
}

// keep = 1 - sigmoid(z) and add = sigmoid(z) * candidate(u): neither loses digits where the gate is near 0 or 1.
// QUICK (the serving precision): the exponential and the reciprocal of the special-function unit, fp32 with an
// error of a few units in the last place; else expf and a division.
template <bool QUICK>
__device__ __forceinline__ void gates(float z, float u, float& keep, float& add) {
    const float e = QUICK ? __expf(-fabsf(z)) : expf(-fabsf(z));
    const float r = QUICK ? __fdividef(1.0f, 1.0f + e) : 1.0f / (1.0f + e);
    const float er = e * r;
    const float open = z >= 0.0f ? r : er;
    keep = z >= 0.0f ? er : r;
    const float f = QUICK ? __expf(fminf(u, 0.0f)) : expf(fminf(u, 0.0f));
    const float low = QUICK ? __fdividef(f, 1.0f + f) : f / (1.0f + f);
    add = open * (u < 0.0f ? low : u + 0.5f);
}
template <bool QUICK>
__device__ __forceinline__ float gate_out(float g) {
    return QUICK ? __fdividef(g, 1.0f + __expf(-g)) : silu_f32(g);
}

struct Shape {
    const float* p;              // projection rows
    long long row_stride;
    int z_col, x_col, g_col;
    const float* z_bias;         // [W] or null
    const float* x_bias;
    float* state;                // [slots][slot_stride], the channels at its head
    long long slot_stride;
    const int* seg_start;
    const int* seg_slot;
    int first_seg, W, ld_out;    // output rows of ld_out >= W entries (zeros behind W)
};

template <int VEC, typename TO>
__global__ void __launch_bounds__(128)
gated_average_step_kernel(const Shape sh, TO* __restrict__ out) {
    fwb::pdl_entry();
    const int seg = sh.first_seg + blockIdx.y;
    const int c = (blockIdx.x * 128 + threadIdx.x) * VEC;
    if (c >= sh.ld_out) return;
    const int t = sh.seg_start[seg];
    TO* dst = out + (size_t)t * sh.ld_out + c;
    Pack<VEC> y;
    if (c >= sh.W) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) y.v[j] = 0.0f;
        store_vec<VEC>(dst, y);
        return;
    }
    const float* row = sh.p + (size_t)t * sh.row_stride + c;
    float* mine = sh.state + (size_t)sh.seg_slot[seg] * sh.slot_stride + c;
    Pack<VEC> z = load_vec<VEC>(row + sh.z_col), u = load_vec<VEC>(row + sh.x_col), g = load_vec<VEC>(row + sh.g_col);
    Pack<VEC> s = load_vec<VEC>(mine);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
        float keep, add;
        gates<quick<TO>()>(z.v[j] + (sh.z_bias ? sh.z_bias[c + j] : 0.0f), u.v[j] + (sh.x_bias ? sh.x_bias[c + j] : 0.0f), keep, add);
        s.v[j] = fmaf(keep, s.v[j], add);
        y.v[j] = s.v[j] * gate_out<quick<TO>()>(g.v[j]);
    }
    store_vec<VEC>(mine, s);
    store_vec<VEC>(dst, y);
}

template <int VEC, typename TO>
__global__ void __launch_bounds__(WARPS * 32, 2)
gated_average_walk_kernel(const Shape sh, TO* __restrict__ out) {
    fwb::pdl_entry();
    constexpr int COLS = 32 * VEC;
    __shared__ __align__(16) float warp_a[WARPS][COLS], warp_b[WARPS][COLS];
    __shared__ __align__(16) float cta_a[2][COLS], cta_b[2][COLS];          // this CTA's stretch, by round parity
    __shared__ __align__(16) float all_a[8][COLS], all_b[8][COLS];          // every CTA's stretch of the round
    cg::cluster_group cluster = cg::this_cluster();
    const int ranks = gridDim.x, rank = blockIdx.x;                          // the cluster spans the grid's x
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int seg = sh.first_seg + blockIdx.z;
    const int c = blockIdx.y * COLS + lane * VEC;
    const bool live = c < sh.W;
    const int first = sh.seg_start[seg], last = sh.seg_start[seg + 1];
    float* mine = sh.state + (size_t)sh.seg_slot[seg] * sh.slot_stride + c;
    Pack<VEC> s, zb, xb;
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
        s.v[j] = live ? mine[j] : 0.0f;
        zb.v[j] = live && sh.z_bias ? sh.z_bias[c + j] : 0.0f;
        xb.v[j] = live && sh.x_bias ? sh.x_bias[c + j] : 0.0f;
    }
    int parity = 0;
    for (int base = first; base < last; base += ranks * STRETCH, parity ^= 1) {
        const int t0 = base + rank * STRETCH + warp * TOKENS;
        Pack<VEC> a[TOKENS], b[TOKENS];
#pragma unroll
        for (int i = 0; i < TOKENS; ++i) {
            const bool on = live && t0 + i < last;
            const float* row = sh.p + (size_t)(t0 + i) * sh.row_stride + c;
            if (on) {
                a[i] = load_vec<VEC>(row + sh.z_col);
                b[i] = load_vec<VEC>(row + sh.x_col);
            } else {
#pragma unroll
                for (int j = 0; j < VEC; ++j) a[i].v[j] = b[i].v[j] = 0.0f;
            }
        }
        Pack<VEC> A, B;                       // this warp's stretch
#pragma unroll
        for (int j = 0; j < VEC; ++j) A.v[j] = 1.0f, B.v[j] = 0.0f;
#pragma unroll
        for (int i = 0; i < TOKENS; ++i) {
            const bool on = t0 + i < last;    // a token that is not there changes nothing: a = 1, b = 0
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
                float keep = 1.0f, add = 0.0f;
                if (on) gates<quick<TO>()>(a[i].v[j] + zb.v[j], b[i].v[j] + xb.v[j], keep, add);
                a[i].v[j] = keep;
                b[i].v[j] = add;
                A.v[j] *= keep;
                B.v[j] = fmaf(keep, B.v[j], add);
            }
        }
        store_vec<VEC>(&warp_a[warp][lane * VEC], A);
        store_vec<VEC>(&warp_b[warp][lane * VEC], B);
        __syncthreads();
        // what the CTA's warps in front of this one make of a state
        Pack<VEC> PA, PB;
#pragma unroll
        for (int j = 0; j < VEC; ++j) PA.v[j] = 1.0f, PB.v[j] = 0.0f;
#pragma unroll 5
        for (int w = 0; w < warp; ++w) {
            const Pack<VEC> wa = load_vec<VEC>(&warp_a[w][lane * VEC]), wb = load_vec<VEC>(&warp_b[w][lane * VEC]);
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
                PB.v[j] = fmaf(wa.v[j], PB.v[j], wb.v[j]);
                PA.v[j] *= wa.v[j];
            }
        }
        if (warp == WARPS - 1) {
            Pack<VEC> CA, CB;
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
                CA.v[j] = A.v[j] * PA.v[j];
                CB.v[j] = fmaf(A.v[j], PB.v[j], B.v[j]);
            }
            store_vec<VEC>(&cta_a[parity][lane * VEC], CA);
            store_vec<VEC>(&cta_b[parity][lane * VEC], CB);
        }
        // the first half's output gates are on their way while the cluster meets
        Pack<VEC> g[TOKENS / 2];
        auto load_gates = [&](int half) {
#pragma unroll
            for (int i = 0; i < TOKENS / 2; ++i) {
                const int t = t0 + half * (TOKENS / 2) + i;
                if (live && t < last) {
                    g[i] = load_vec<VEC>(sh.p + (size_t)t * sh.row_stride + c + sh.g_col);
                } else {
#pragma unroll
                    for (int j = 0; j < VEC; ++j) g[i].v[j] = 0.0f;
                }
            }
        };
        load_gates(0);
        cluster.sync();
        // one warp fetches one CTA's stretch: a single trip through distributed shared memory
        if (warp < ranks) {
            store_vec<VEC>(&all_a[warp][lane * VEC], load_vec<VEC>(cluster.map_shared_rank(&cta_a[parity][lane * VEC], warp)));
            store_vec<VEC>(&all_b[warp][lane * VEC], load_vec<VEC>(cluster.map_shared_rank(&cta_b[parity][lane * VEC], warp)));
        }
        __syncthreads();
        // the state in front of this CTA's stretch, and the one behind the round
        Pack<VEC> front = s;
#pragma unroll 4
        for (int r = 0; r < ranks; ++r) {
            if (r == rank) front = s;
            const Pack<VEC> ra = load_vec<VEC>(&all_a[r][lane * VEC]), rb = load_vec<VEC>(&all_b[r][lane * VEC]);
#pragma unroll
            for (int j = 0; j < VEC; ++j) s.v[j] = fmaf(ra.v[j], s.v[j], rb.v[j]);
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) front.v[j] = fmaf(PA.v[j], front.v[j], PB.v[j]);
#pragma unroll
        for (int i = 0; i < TOKENS; ++i) {
            if (i == TOKENS / 2) load_gates(1);
            Pack<VEC> y;
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
                front.v[j] = fmaf(a[i].v[j], front.v[j], b[i].v[j]);
                y.v[j] = live ? front.v[j] * gate_out<quick<TO>()>(g[i % (TOKENS / 2)].v[j]) : 0.0f;
            }
            if (t0 + i < last && c < sh.ld_out) store_vec<VEC>(out + (size_t)(t0 + i) * sh.ld_out + c, y);
        }
        // (the next round writes warp_a / warp_b behind this round's cluster barrier, which every warp reached
        // after reading them, the other parity's cta_a / cta_b, and all_a / all_b behind its own barriers)
    }
    cluster.sync();                            // nobody leaves while a peer may still read its stretch
    if (rank == 0 && warp == 0 && live) store_vec<VEC>(mine, s);
}

template <int VEC, typename TO>
int launch_walk(const Shape& sh, TO* out, int segments, int ranks, cudaStream_t stream) {
    cudaLaunchConfig_t config = {};
    config.gridDim = dim3(ranks, (sh.ld_out + 32 * VEC - 1) / (32 * VEC), segments);
    config.blockDim = dim3(WARPS * 32);
    config.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = ranks;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    config.attrs = attr;
    config.numAttrs = pdl_enabled() ? 2 : 1;
    cudaError_t e = cudaLaunchKernelEx(&config, gated_average_walk_kernel<VEC, TO>, sh, out);
    return e == cudaSuccess ? fwb_launch_status() : (int)e;
}

template <typename TO>
int run(const Shape& sh, TO* out, int segments, int max_segment, int vec, cudaStream_t stream) {
    if (max_segment == 1) {
        const dim3 grid((sh.ld_out + 128 * vec - 1) / (128 * vec), segments);
        if (vec == 4) fwb::pdl(gated_average_step_kernel<4, TO>, grid, 128, 0, stream)(sh, out);
        else if (vec == 2) fwb::pdl(gated_average_step_kernel<2, TO>, grid, 128, 0, stream)(sh, out);
        else fwb::pdl(gated_average_step_kernel<1, TO>, grid, 128, 0, stream)(sh, out);
        return fwb_launch_status();
    }
    int ranks = 1;
    while (ranks < 8 && ranks * STRETCH < max_segment) ranks *= 2;
    // (two channels a lane: with four, a warp's eight tokens do not fit the registers of two CTAs an SM)
    if (vec >= 2) return launch_walk<2, TO>(sh, out, segments, ranks, stream);
    return launch_walk<1, TO>(sh, out, segments, ranks, stream);
}

}  // namespace

// p: fp32 rows of `row_stride` entries, one per token, whose columns from z_col, x_col and g_col (W each) are
// the projections.  z_bias, x_bias: fp32 [W] or null.  state: fp32, a request's slot `slot_stride` entries
// after the one before, [W] at its head (read at the head of every segment and advanced).  The step's segments
// first_seg .. first_seg + segments - 1 run, each of at most `max_segment` tokens (1: the one-token form, which
// takes a segment's first token only).  out: [T][ld_out] fp32 or bf16, ld_out >= W, zeros behind column W.
FWB_API int fwb_gated_average(const float* p, long long row_stride, int z_col, int x_col, int g_col,
                              const float* z_bias, const float* x_bias, float* state, long long slot_stride,
                              const int* seg_start, const int* seg_slot, int first_seg, int segments,
                              int max_segment, void* out, int out_bf16, int W, int ld_out, cudaStream_t stream) {
    if (segments <= 0 || max_segment <= 0) return FWB_OK;
    if (!p || !state || !seg_start || !seg_slot || !out) return FWB_BAD_ARGUMENT;
    if (W <= 0 || ld_out < W || z_col < 0 || x_col < 0 || g_col < 0 || first_seg < 0 || row_stride < W || slot_stride < W)
        return FWB_BAD_ARGUMENT;
    if (segments > 65535 || ld_out > 65535 * 32) return FWB_TOO_LARGE;
    const Shape sh{p, row_stride, z_col, x_col, g_col, z_bias, x_bias, state, slot_stride, seg_start, seg_slot,
                   first_seg, W, ld_out};
    // the widest access that every row, column and slot starts aligned to
    int vec = 4;
    while (vec > 1 && (W % vec || ld_out % vec || row_stride % vec || z_col % vec || x_col % vec || g_col % vec ||
                       slot_stride % vec || (uintptr_t)p % (4 * vec) || (uintptr_t)state % (4 * vec) ||
                       (uintptr_t)out % (4 * vec)))
        vec /= 2;
    if (out_bf16) return run<__nv_bfloat16>(sh, (__nv_bfloat16*)out, segments, max_segment, vec, stream);
    return run<float>(sh, (float*)out, segments, max_segment, vec, stream);
}
