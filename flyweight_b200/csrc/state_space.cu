// A state-space recurrence with one scalar decay per head and token (Mamba-2): the state is one [n][e] matrix
// per head and request, kept in fp32 in the request's slot.
//
//   dt_t = softplus(raw_t + dt_bias_h),   S_t = exp(-exp(a_log_h) dt_t) S_(t-1) + dt_t b_t x_t^T,
//   y_t = S_t^T c_t + skip_h x_t
//
// x (H heads of e channels), b and c (G groups of n channels; head h reads group h / (H/G)) are columns of one
// row buffer `u` per token, x | b | c, which has passed its convolution; raw is a column per head of the fp32
// projection.  Step sizes, decays, their sums, the state and every accumulation are fp32.
//
//   fwb_state_scan   token by token, any sizes, fp32 arithmetic: single tokens, and the 32-bit path.  One block
//                    owns 32 columns of one head's state for one segment; the state's rows are cut over the
//                    block's warps, 16 rows a thread, in registers.  A token's arithmetic is the same whatever
//                    the cut of the sequence into steps.
//   fwb_state_runs   portions of prompts in bfloat16, 64 tokens at a time on tensor cores (below)
//   fwb_gate_group_norm   out = weight * unit(y * silu(z)), unit over each of equal runs of channels
#include "common.cuh"

using namespace fwb;

namespace {

constexpr int COLS = 32;      // scan: state columns per block (one per lane)
constexpr int ROWS = 16;      // scan: state rows per thread
constexpr int STAGE = 16;     // scan: tokens staged at a time
constexpr int MAX_SPLITS = 32;

__device__ __forceinline__ float softplus_f32(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

template <typename TU>
__global__ void __launch_bounds__(COLS * MAX_SPLITS)
state_scan_kernel(const TU* __restrict__ u, long long u_stride, const float* __restrict__ raw, long long raw_stride,
                  const float* __restrict__ dt_bias, const float* __restrict__ a_log, const float* __restrict__ skip,
                  float* __restrict__ state, long long slot_stride, const int* __restrict__ seg_start,
                  const int* __restrict__ seg_slot, float* __restrict__ y, int first_seg, int H, int G, int n, int e) {
    fwb::pdl_entry();
    extern __shared__ float smem[];
    const int splits = blockDim.x / COLS, npad = splits * ROWS;
    float* bs = smem;                          // [STAGE][npad]  b
    float* cs = bs + STAGE * npad;             // [STAGE][npad]  c
    float* xs = cs + STAGE * npad;             // [STAGE][COLS]
    float* step = xs + STAGE * COLS;           // [STAGE]  dt
    float* decay = step + STAGE;               // [STAGE]
    float* part = decay + STAGE;               // [splits][STAGE][COLS]
    const int seg = first_seg + blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * COLS;
    const int el = threadIdx.x & (COLS - 1), ds = threadIdx.x / COLS;
    const int col = e0 + el;
    const bool live = col < e;
    const int first = seg_start[seg], last = seg_start[seg + 1];
    const int group = h / (H / G);
    const int x_col = h * e, b_col = H * e + group * n, c_col = b_col + G * n;
    const float a = expf(a_log[h]), bias = dt_bias[h], d = skip[h];
    float* mine = state + (size_t)seg_slot[seg] * slot_stride + (size_t)h * n * e;

    float s[ROWS];
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        const int row = ds * ROWS + j;
        s[j] = (live && row < n) ? mine[(size_t)row * e + col] : 0.0f;
    }
    for (int t0 = first; t0 < last; t0 += STAGE) {
        const int count = last - t0 < STAGE ? last - t0 : STAGE;
        __syncthreads();
        for (int i = threadIdx.x; i < count * npad; i += blockDim.x) {
            const int tok = i / npad, row = i - tok * npad;
            const TU* src = u + (size_t)(t0 + tok) * u_stride + row;
            bs[i] = row < n ? to_f32<TU>(src[b_col]) : 0.0f;
            cs[i] = row < n ? to_f32<TU>(src[c_col]) : 0.0f;
        }
        for (int i = threadIdx.x; i < count * COLS; i += blockDim.x) {
            const int tok = i / COLS, c = e0 + (i - tok * COLS);
            xs[i] = c < e ? to_f32<TU>(u[(size_t)(t0 + tok) * u_stride + x_col + c]) : 0.0f;
        }
        for (int tok = threadIdx.x; tok < count; tok += blockDim.x) {
            const float dt = softplus_f32(raw[(size_t)(t0 + tok) * raw_stride + h] + bias);
            step[tok] = dt;
            decay[tok] = expf(-a * dt);
        }
        __syncthreads();
        for (int tok = 0; tok < count; ++tok) {
            const float v = xs[tok * COLS + el] * step[tok], g = decay[tok];
            const float* br = bs + tok * npad + ds * ROWS;
            const float* cr = cs + tok * npad + ds * ROWS;
            float a0 = 0.0f, a1 = 0.0f;
#pragma unroll
            for (int j = 0; j < ROWS; j += 2) {
                s[j] = fmaf(g, s[j], br[j] * v);
                s[j + 1] = fmaf(g, s[j + 1], br[j + 1] * v);
                a0 = fmaf(s[j], cr[j], a0);
                a1 = fmaf(s[j + 1], cr[j + 1], a1);
            }
            part[(ds * STAGE + tok) * COLS + el] = a0 + a1;
        }
        __syncthreads();
        for (int i = threadIdx.x; i < count * COLS; i += blockDim.x) {
            const int tok = i / COLS, c = i - tok * COLS;
            if (e0 + c >= e) continue;
            float sum = 0.0f;
            for (int w = 0; w < splits; ++w) sum += part[(w * STAGE + tok) * COLS + c];
            y[(size_t)(t0 + tok) * H * e + (size_t)h * e + e0 + c] = fmaf(d, xs[i], sum);
        }
    }
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        const int row = ds * ROWS + j;
        if (live && row < n) mine[(size_t)row * e + col] = s[j];
    }
}

// ---------------------------------------------------------------------------------------------------
// Portions of prompts, 64 tokens at a time on tensor cores (the serving path in bfloat16).  With S the state
// in front of a run of m tokens and L_i = sum of the logarithms of the decays of tokens 0 .. i of the run,
//
//   y_i = exp(L_i) S^T c_i + sum_{j <= i} exp(L_i - L_j) dt_j (c_i . b_j) x_j + skip x_i
//   S'  = exp(L_(m-1)) S + sum_j b_j (exp(L_(m-1) - L_j) dt_j x_j)^T
//
// One block owns 64 columns of one head's state for one piece of a segment and walks its runs in order.  x, b
// and c are bfloat16 as their convolution left them; step sizes, logarithms, decays, scores and the state are
// fp32, and wherever an fp32 quantity is an operand of a product (the state, the decayed scores, the decayed
// values) it enters as the sum of two bfloat16 numbers, two products into one fp32 accumulator.  The state
// lives in the accumulators of the update's product (a warp owns 16 of its rows, or two such bands).
//
// A long segment is cut into pieces of `piece_len` tokens (a multiple of 64) that run side by side: a first
// launch sums what each piece alone adds to a zero state and its total decay, a small kernel chains those into
// the state in front of every piece, and the main launch walks every piece from its own start.  Only a
// segment's last piece writes the slot.
constexpr int RUN = 64;
constexpr int CT = 64;             // state columns per block
constexpr int VS = CT + 8;         // bf16 entries of a shared row of columns
constexpr int THREADS = 256;       // eight warps: four bands of 16 tokens by two halves of the columns
constexpr int MAX_STATE = 256;

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// the two halves x = hi + lo, hi = bf16(x), of a pair of fp32 operands
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h2 = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 l2 = __floats2bfloat162_rn(x - __low2float(h2), y - __high2float(h2));
    hi = *reinterpret_cast<const uint32_t*>(&h2);
    lo = *reinterpret_cast<const uint32_t*>(&l2);
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
__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
    const uint32_t s = static_cast<uint32_t>(__cvta_generic_to_shared(smem));
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem) : "memory");
}

// RUN rows of `width` channels (zero padding up to `padded`) into shared rows `ld` entries apart; rows from
// `count` on are zero.  VEC: 16-byte copies (the caller has checked widths and alignment).
template <bool VEC>
__device__ __forceinline__ void load_rows(__nv_bfloat16* dst, int ld, const __nv_bfloat16* __restrict__ src,
                                          long long stride, int count, int width, int padded) {
    if constexpr (VEC) {
        const int chunks = padded >> 3, tok_step = THREADS / chunks, chunk_step = THREADS % chunks;
        for (int tok = threadIdx.x / chunks, c = threadIdx.x % chunks; tok < RUN;) {
            __nv_bfloat16* at = dst + tok * ld + c * 8;
            if (tok < count && c * 8 < width) cp_async16(at, src + tok * stride + c * 8);
            else *reinterpret_cast<uint4*>(at) = make_uint4(0u, 0u, 0u, 0u);
            tok += tok_step;
            c += chunk_step;
            if (c >= chunks) {
                c -= chunks;
                ++tok;
            }
        }
    } else {
        for (int i = threadIdx.x; i < RUN * padded; i += THREADS) {
            const int tok = i / padded, c = i - tok * padded;
            dst[tok * ld + c] = (tok < count && c < width) ? src[(size_t)tok * stride + c] : __float2bfloat16_rn(0.0f);
        }
    }
}

// SUMS: the first launch (what a piece adds to a zero state, and the logarithm of its total decay).
// MT: bands of 128 state rows (16 a warp).
template <bool SUMS, bool VEC, int MT>
__global__ void __launch_bounds__(THREADS, MT == 1 ? 2 : 1)
state_runs_kernel(const __nv_bfloat16* __restrict__ u, long long u_stride, const float* __restrict__ raw,
                  long long raw_stride, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                  const float* __restrict__ skip, float* __restrict__ state, long long slot_stride,
                  const int* __restrict__ seg_start, const int* __restrict__ seg_slot,
                  const int* __restrict__ piece_seg, const int* __restrict__ piece_tok0, int piece_len,
                  float* __restrict__ scratch, float* __restrict__ scratch_log, float* __restrict__ y, int H, int G,
                  int n, int e, int NP) {
    fwb::pdl_entry();
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const int NS = NP + 8;
    __nv_bfloat16* Bs = reinterpret_cast<__nv_bfloat16*>(smem_raw);     // [RUN][NS]
    __nv_bfloat16* Cs = Bs + RUN * NS;                                  // [RUN][NS]
    __nv_bfloat16* Xs = Cs + RUN * NS;                                  // [RUN][VS]
    __nv_bfloat16* Vhi = Xs + RUN * VS;                                 // [RUN][VS]  decayed values, two halves
    __nv_bfloat16* Vlo = Vhi + RUN * VS;
    __nv_bfloat16* Shi = Vlo + RUN * VS;                                // [NP][VS]   the state, two halves
    __nv_bfloat16* Slo = Shi + NP * VS;
    float* logs = reinterpret_cast<float*>(Slo + NP * VS);              // [RUN]  L_i
    float* steps = logs + RUN;                                          // [RUN]  dt_i
    float* into = steps + RUN;                                          // [RUN]  exp(L_i)
    float* onto = into + RUN;                                           // [RUN]  exp(L_last - L_j) dt_j

    const int piece = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * CT;
    const int seg = piece_seg[piece], first = piece_tok0[piece], seg_end = seg_start[seg + 1];
    const int last = first + piece_len < seg_end ? first + piece_len : seg_end;
    const bool head = first == seg_start[seg], tail = last == seg_end;
    if (SUMS && tail) return;                          // nothing follows this piece: its sum is not needed
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int n16 = NP >> 4;
    const int group = h / (H / G);
    const int live_cols = e - e0 < CT ? e - e0 : CT;
    const float a = expf(a_log[h]), bias = dt_bias[h], d = skip[h];
    const size_t head_at = (size_t)h * n * e;
    float* mine = state + (size_t)seg_slot[seg] * slot_stride + head_at;
    float* held = scratch ? scratch + (size_t)piece * H * n * e + head_at : nullptr;
    // the state in front of the piece: the slot's for a segment of one piece, else what the chain left
    const float* front = SUMS ? nullptr : (head && tail ? mine : held);
    float* behind = SUMS ? held : (tail ? mine : nullptr);
    float total = 0.0f;                                // logarithm of the piece's decay so far (warp 0)
    // warp 0 turns a run's step inputs into decays; it asks for them one run ahead
    float ahead[2];
    auto ask = [&](int t0) {
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int tok = t0 + lane + 32 * k;
            ahead[k] = tok < last ? raw[(size_t)tok * raw_stride + h] : 0.0f;
        }
    };
    if (warp == 0) ask(first);

    float S[MT][CT / 8][4];                            // rows (mt*8 + warp)*16 + g (+8), columns nt*8 + 2t (+1)
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < CT / 8; ++nt)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int r = (mt * 8 + warp) * 16 + g + 8 * (j >> 1), c = nt * 8 + 2 * t + (j & 1);
                S[mt][nt][j] = (front && r < n && c < live_cols) ? front[(size_t)r * e + e0 + c] : 0.0f;
            }

    for (int t0 = first; t0 < last; t0 += RUN) {
        const int m = last - t0 < RUN ? last - t0 : RUN;
        __syncthreads();                               // the run before is done with the shared rows
        const __nv_bfloat16* row0 = u + (size_t)t0 * u_stride;
        load_rows<VEC>(Bs, NS, row0 + (size_t)H * e + group * n, u_stride, m, n, NP);
        if (!SUMS) load_rows<VEC>(Cs, NS, row0 + (size_t)H * e + (G + group) * n, u_stride, m, n, NP);
        load_rows<VEC>(Xs, VS, row0 + h * e + e0, u_stride, m, live_cols, CT);
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (warp == 0) {
            float dt[2], sum[2];
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int tok = lane + 32 * k;
                dt[k] = tok < m ? softplus_f32(ahead[k] + bias) : 0.0f;
                sum[k] = -a * dt[k];
            }
            ask(t0 + RUN);
#pragma unroll
            for (int step = 1; step < 32; step <<= 1)
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    const float before = __shfl_up_sync(0xffffffffu, sum[k], step);
                    if (lane >= step) sum[k] += before;
                }
            sum[1] += __shfl_sync(0xffffffffu, sum[0], 31);
            const float whole = __shfl_sync(0xffffffffu, sum[1], 31);
            total += whole;
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int tok = lane + 32 * k;
                logs[tok] = sum[k];
                steps[tok] = dt[k];
                into[tok] = expf(sum[k]);
                onto[tok] = expf(whole - sum[k]) * dt[k];
            }
        }
        if (!SUMS) {
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
                const int r = (mt * 8 + warp) * 16 + g;
                if (r - g >= NP) break;
#pragma unroll
                for (int nt = 0; nt < CT / 8; ++nt)
#pragma unroll
                    for (int half = 0; half < 2; ++half) {
                        uint32_t hi, lo;
                        split_pair(S[mt][nt][2 * half], S[mt][nt][2 * half + 1], hi, lo);
                        const int at = (r + 8 * half) * VS + nt * 8 + 2 * t;
                        *reinterpret_cast<uint32_t*>(Shi + at) = hi;
                        *reinterpret_cast<uint32_t*>(Slo + at) = lo;
                    }
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        for (int i = tid; i < RUN * CT / 4; i += THREADS) {
            const int tok = i / (CT / 4), c = (i % (CT / 4)) << 2;
            const uint2 raw2 = *reinterpret_cast<const uint2*>(Xs + tok * VS + c);
            const __nv_bfloat162 x01 = *reinterpret_cast<const __nv_bfloat162*>(&raw2.x);
            const __nv_bfloat162 x23 = *reinterpret_cast<const __nv_bfloat162*>(&raw2.y);
            const float w = onto[tok];
            uint2 hi, lo;
            split_pair(__low2float(x01) * w, __high2float(x01) * w, hi.x, lo.x);
            split_pair(__low2float(x23) * w, __high2float(x23) * w, hi.y, lo.y);
            *reinterpret_cast<uint2*>(Vhi + tok * VS + c) = hi;
            *reinterpret_cast<uint2*>(Vlo + tok * VS + c) = lo;
        }
        // the address this lane gives to a transposing load of 16 rows by 16 columns (values, state)
        const int v_lane = (lane & 15) * VS + ((lane >> 4) << 3);
        const int band = warp & 3, tok0 = band * 16, col0 = (warp >> 2) * 32;
        if (!SUMS && tok0 < m && col0 < live_cols) {
            float acc[4][4];
#pragma unroll
            for (int nt = 0; nt < 4; ++nt)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[nt][j] = 0.0f;
            const __nv_bfloat16* ca = Cs + (tok0 + (lane & 15)) * NS + ((lane >> 4) << 3);
            for (int ks = 0; ks < n16; ++ks) {
                uint32_t q[4];
                ldsm4(q, ca + ks * 16);
#pragma unroll
                for (int np = 0; np < 2; ++np) {
                    uint32_t b[4];
                    ldsm4t(b, Shi + ks * 16 * VS + col0 + np * 16 + v_lane);
                    mma_bf16(acc[2 * np], q, b[0], b[1]);
                    mma_bf16(acc[2 * np + 1], q, b[2], b[3]);
                    ldsm4t(b, Slo + ks * 16 * VS + col0 + np * 16 + v_lane);
                    mma_bf16(acc[2 * np], q, b[0], b[1]);
                    mma_bf16(acc[2 * np + 1], q, b[2], b[3]);
                }
            }
            const float up = into[tok0 + g], down = into[tok0 + g + 8];
            const float l_up = logs[tok0 + g], l_down = logs[tok0 + g + 8];
#pragma unroll
            for (int nt = 0; nt < 4; ++nt) {
                acc[nt][0] *= up;
                acc[nt][1] *= up;
                acc[nt][2] *= down;
                acc[nt][3] *= down;
            }
            // the run's own tokens, 16 at a time up to this warp's last one
            const __nv_bfloat16* kb = Bs + ((lane & 7) + ((lane >> 4) << 3)) * NS + (((lane >> 3) & 1) << 3);
            for (int kk = 0; kk <= band; ++kk) {
                float sc[2][4] = {{0.0f, 0.0f, 0.0f, 0.0f}, {0.0f, 0.0f, 0.0f, 0.0f}};
                for (int ks = 0; ks < n16; ++ks) {
                    uint32_t q[4], b[4];
                    ldsm4(q, ca + ks * 16);
                    ldsm4(b, kb + kk * 16 * NS + ks * 16);
                    mma_bf16(sc[0], q, b[0], b[1]);
                    mma_bf16(sc[1], q, b[2], b[3]);
                }
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int j = kk * 16 + half * 8 + 2 * t;
                    const float2 lj = *reinterpret_cast<const float2*>(logs + j);
                    const float2 dj = *reinterpret_cast<const float2*>(steps + j);
#pragma unroll
                    for (int rr = 0; rr < 2; ++rr) {
                        const int i = tok0 + g + 8 * rr;
                        const float li = rr ? l_down : l_up;
                        const float w0 = j <= i ? sc[half][2 * rr] * (__expf(li - lj.x) * dj.x) : 0.0f;
                        const float w1 = j + 1 <= i ? sc[half][2 * rr + 1] * (__expf(li - lj.y) * dj.y) : 0.0f;
                        split_pair(w0, w1, hi[2 * half + rr], lo[2 * half + rr]);
                    }
                }
#pragma unroll
                for (int np = 0; np < 2; ++np) {
                    uint32_t b[4];
                    ldsm4t(b, Xs + kk * 16 * VS + col0 + np * 16 + v_lane);
                    mma_bf16(acc[2 * np], hi, b[0], b[1]);
                    mma_bf16(acc[2 * np], lo, b[0], b[1]);
                    mma_bf16(acc[2 * np + 1], hi, b[2], b[3]);
                    mma_bf16(acc[2 * np + 1], lo, b[2], b[3]);
                }
            }
#pragma unroll
            for (int nt = 0; nt < 4; ++nt)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int i = tok0 + g + 8 * half, c = col0 + nt * 8 + 2 * t;
                    if (i >= m || c >= live_cols) continue;
                    const __nv_bfloat162 x2 = *reinterpret_cast<const __nv_bfloat162*>(Xs + i * VS + c);
                    const float v0 = fmaf(d, __low2float(x2), acc[nt][2 * half]);
                    const float v1 = fmaf(d, __high2float(x2), acc[nt][2 * half + 1]);
                    float* dst = y + (size_t)(t0 + i) * H * e + (size_t)h * e + e0 + c;
                    if (VEC) {
                        *reinterpret_cast<float2*>(dst) = make_float2(v0, v1);
                    } else {
                        dst[0] = v0;
                        if (c + 1 < live_cols) dst[1] = v1;
                    }
                }
        }
        __syncthreads();                               // the decayed values are in place
        const float shrink = into[RUN - 1];            // tokens behind the run's last have the decay 1
        const int k16 = (m + 15) >> 4;
        // this lane's address in a transposing load of b: 16 tokens by 16 channels
        const int k_lane = ((lane & 7) + ((lane >> 4) << 3)) * NS + (((lane >> 3) & 1) << 3);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
            const int r0 = (mt * 8 + warp) * 16;
            if (r0 >= NP) break;
#pragma unroll
            for (int nt = 0; nt < CT / 8; ++nt)
#pragma unroll
                for (int j = 0; j < 4; ++j) S[mt][nt][j] *= shrink;
            for (int ks = 0; ks < k16; ++ks) {
                uint32_t k[4];
                ldsm4t(k, Bs + ks * 16 * NS + r0 + k_lane);
#pragma unroll
                for (int np = 0; np < CT / 16; ++np) {
                    uint32_t b[4];
                    ldsm4t(b, Vhi + ks * 16 * VS + np * 16 + v_lane);
                    mma_bf16(S[mt][2 * np], k, b[0], b[1]);
                    mma_bf16(S[mt][2 * np + 1], k, b[2], b[3]);
                    ldsm4t(b, Vlo + ks * 16 * VS + np * 16 + v_lane);
                    mma_bf16(S[mt][2 * np], k, b[0], b[1]);
                    mma_bf16(S[mt][2 * np + 1], k, b[2], b[3]);
                }
            }
        }
    }
    if (SUMS && warp == 0 && lane == 0 && blockIdx.z == 0) scratch_log[(size_t)piece * H + h] = total;
    if (!behind) return;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < CT / 8; ++nt)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int r = (mt * 8 + warp) * 16 + g + 8 * (j >> 1), c = nt * 8 + 2 * t + (j & 1);
                if (r < n && c < live_cols) behind[(size_t)r * e + e0 + c] = S[mt][nt][j];
            }
}

// Chains the pieces' sums: walking a segment's pieces in order, every piece's entry of `scratch` (what the
// piece alone adds) is replaced by the state in front of that piece.  One thread per state entry; blocks of
// pieces that are not the first of a segment of several pieces have nothing to do.
__global__ void __launch_bounds__(256)
state_chain_kernel(const float* __restrict__ state, long long slot_stride, const int* __restrict__ seg_start,
                   const int* __restrict__ seg_slot, const int* __restrict__ piece_seg,
                   const int* __restrict__ piece_tok0, int piece_len, float* __restrict__ scratch,
                   const float* __restrict__ scratch_log, int H, int per_head) {
    fwb::pdl_entry();
    const int piece = blockIdx.x;
    const int seg = piece_seg[piece], first = piece_tok0[piece], seg_end = seg_start[seg + 1];
    if (first != seg_start[seg] || first + piece_len >= seg_end) return;
    const size_t size = (size_t)H * per_head;
    const size_t at = (size_t)blockIdx.y * blockDim.x + threadIdx.x;
    if (at >= size) return;
    const int h = (int)(at / per_head);
    float run = state[(size_t)seg_slot[seg] * slot_stride + at];
    for (int c = piece;; ++c) {
        float* cell = scratch + (size_t)c * size + at;
        if (piece_tok0[c] + piece_len >= seg_end) {        // the segment's last piece
            *cell = run;
            break;
        }
        const float sum = *cell, shrink = expf(scratch_log[(size_t)c * H + h]);
        *cell = run;
        run = fmaf(shrink, run, sum);
    }
}

size_t state_runs_smem(int NP) {
    return (size_t)(2 * RUN * (NP + 8) + 3 * RUN * VS + 2 * NP * VS) * sizeof(__nv_bfloat16) + 4 * RUN * sizeof(float);
}

// One block per (token, run of channels): v = y silu(z), out = weight v / sqrt(mean(v^2) + eps).
template <typename TO>
__global__ void __launch_bounds__(256)
gate_group_norm_kernel(const float* __restrict__ y, const float* __restrict__ z, long long z_stride,
                       const float* __restrict__ weight, float eps, TO* __restrict__ out, int width, int part) {
    fwb::pdl_entry();
    extern __shared__ float row[];                 // [part]
    __shared__ float scratch[33];
    const int t = blockIdx.x, c0 = blockIdx.y * part;
    const float* yr = y + (size_t)t * width + c0;
    const float* zr = z + (size_t)t * z_stride + c0;
    float ss = 0.0f;
    if ((part & 3) == 0 && (width & 3) == 0 && (z_stride & 3) == 0 && (((uintptr_t)y | (uintptr_t)z) & 15) == 0) {
        for (int c = 4 * threadIdx.x; c < part; c += 4 * blockDim.x) {
            const float4 a = *reinterpret_cast<const float4*>(yr + c), b = *reinterpret_cast<const float4*>(zr + c);
            const float4 v = make_float4(a.x * silu_f32(b.x), a.y * silu_f32(b.y), a.z * silu_f32(b.z), a.w * silu_f32(b.w));
            *reinterpret_cast<float4*>(row + c) = v;
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        }
    } else {
        for (int c = threadIdx.x; c < part; c += blockDim.x) {
            const float v = yr[c] * silu_f32(zr[c]);
            row[c] = v;
            ss = fmaf(v, v, ss);
        }
    }
    const float inv = rsqrtf(block_sum(ss, scratch) / (float)part + eps);      // (its barriers cover `row` too)
    TO* dst = out + (size_t)t * width + c0;
    if constexpr (sizeof(TO) == 2) if (((part | width) & 1) == 0 && ((uintptr_t)out & 3) == 0) {
        for (int c = 2 * threadIdx.x; c < part; c += 2 * blockDim.x) {
            const __nv_bfloat162 v = __floats2bfloat162_rn((row[c] * inv) * weight[c0 + c], (row[c + 1] * inv) * weight[c0 + c + 1]);
            *reinterpret_cast<__nv_bfloat162*>(dst + c) = v;
        }
        return;
    }
    for (int c = threadIdx.x; c < part; c += blockDim.x) dst[c] = from_f32<TO>((row[c] * inv) * weight[c0 + c]);
}

bool sizes_ok(int H, int G, int n, int e, long long u_stride, long long raw_stride, long long slot_stride) {
    return H > 0 && G > 0 && H % G == 0 && n > 0 && e > 0 && u_stride >= (long long)H * e + 2LL * G * n &&
           raw_stride >= H && slot_stride >= (long long)H * n * e;
}

}  // namespace

// u: [T] rows of `u_stride` entries, x [H][e] | b [G][n] | c [G][n], fp32 or bf16.  raw: fp32, entry h of token t
// at raw[t * raw_stride + h].  dt_bias, a_log, skip: fp32 [H].  state: fp32, a request's slot `slot_stride`
// entries after the one before, [H][n][e] at its head (read at the head of every segment and advanced).
// seg_start, seg_slot: the step's segments, of which `S` from `first_seg` on are walked.  y: fp32 [T][H][e].
FWB_API int fwb_state_scan(const void* u, int u_bf16, long long u_stride, const float* raw, long long raw_stride,
                           const float* dt_bias, const float* a_log, const float* skip, float* state,
                           long long slot_stride, const int* seg_start, const int* seg_slot, float* y, int first_seg,
                           int S, int H, int G, int n, int e, cudaStream_t stream) {
    if (S <= 0) return FWB_OK;
    if (!u || !raw || !dt_bias || !a_log || !skip || !state || !seg_start || !seg_slot || !y || first_seg < 0)
        return FWB_BAD_ARGUMENT;
    if (!sizes_ok(H, G, n, e, u_stride, raw_stride, slot_stride)) return FWB_BAD_ARGUMENT;
    const int splits = (n + ROWS - 1) / ROWS, tiles = (e + COLS - 1) / COLS;
    if (splits > MAX_SPLITS || H > 65535 || tiles > 65535) return FWB_TOO_LARGE;
    const size_t smem = ((size_t)2 * STAGE * splits * ROWS + (size_t)STAGE * COLS + 2 * STAGE
                         + (size_t)splits * STAGE * COLS) * sizeof(float);
    auto launch = [&](auto kernel, auto rows) -> int {
        if (smem > 48 * 1024) {
            cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (err != cudaSuccess) return (int)err;
        }
        fwb::pdl(kernel, dim3(S, H, tiles), COLS * splits, smem, stream)(
            rows, u_stride, raw, raw_stride, dt_bias, a_log, skip, state, slot_stride, seg_start, seg_slot, y, first_seg,
            H, G, n, e);
        return fwb_launch_status();
    };
    return u_bf16 ? launch(state_scan_kernel<__nv_bfloat16>, (const __nv_bfloat16*)u)
                  : launch(state_scan_kernel<float>, (const float*)u);
}

// The same operation for portions of prompts, u bf16, states of up to 256 rows (FWB_UNSUPPORTED beyond: the scan
// takes those).  The segments come cut into `P` pieces of at most `piece_len` tokens (a multiple of 64):
// piece_seg, piece_tok0 (segments that no piece names are left alone).  scratch: fp32 [P][H n e], scratch_log:
// fp32 [P][H], needed when some segment has more than one piece (`chained` != 0), else they may be null.
FWB_API int fwb_state_runs(const void* u, long long u_stride, const float* raw, long long raw_stride,
                           const float* dt_bias, const float* a_log, const float* skip, float* state,
                           long long slot_stride, const int* seg_start, const int* seg_slot, const int* piece_seg,
                           const int* piece_tok0, int piece_len, int chained, float* scratch, float* scratch_log,
                           float* y, int P, int H, int G, int n, int e, cudaStream_t stream) {
    if (P <= 0) return FWB_OK;
    if (!u || !raw || !dt_bias || !a_log || !skip || !state || !seg_start || !seg_slot || !piece_seg || !piece_tok0 || !y)
        return FWB_BAD_ARGUMENT;
    if (piece_len <= 0 || piece_len % RUN != 0 || (chained && (!scratch || !scratch_log))) return FWB_BAD_ARGUMENT;
    if (!sizes_ok(H, G, n, e, u_stride, raw_stride, slot_stride)) return FWB_BAD_ARGUMENT;
    if (n > MAX_STATE) return FWB_UNSUPPORTED;
    const int tiles = (e + CT - 1) / CT;
    const size_t size = (size_t)H * n * e;
    if (H > 65535 || tiles > 65535 || (size + 255) / 256 > 65535) return FWB_TOO_LARGE;
    const int NP = (n + 15) / 16 * 16;
    const size_t smem = state_runs_smem(NP);
    const bool vec = n % 8 == 0 && e % 8 == 0 && u_stride % 8 == 0 && reinterpret_cast<uintptr_t>(u) % 16 == 0;
    auto run = [&](auto kernel) -> int {
        cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (err != cudaSuccess) return (int)err;
        fwb::pdl(kernel, dim3(P, H, tiles), THREADS, smem, stream)(
            (const __nv_bfloat16*)u, u_stride, raw, raw_stride, dt_bias, a_log, skip, state, slot_stride, seg_start,
            seg_slot, piece_seg, piece_tok0, piece_len, chained ? scratch : nullptr, scratch_log, y, H, G, n, e, NP);
        return fwb_launch_status();
    };
    int status = FWB_OK;
    if (chained) {
        status = NP <= 128 ? (vec ? run(state_runs_kernel<true, true, 1>) : run(state_runs_kernel<true, false, 1>))
                           : (vec ? run(state_runs_kernel<true, true, 2>) : run(state_runs_kernel<true, false, 2>));
        if (status != FWB_OK) return status;
        fwb::pdl(state_chain_kernel, dim3(P, (unsigned)((size + 255) / 256)), 256, 0, stream)(
            state, slot_stride, seg_start, seg_slot, piece_seg, piece_tok0, piece_len, scratch, scratch_log, H, n * e);
        status = fwb_launch_status();
        if (status != FWB_OK) return status;
    }
    return NP <= 128 ? (vec ? run(state_runs_kernel<false, true, 1>) : run(state_runs_kernel<false, false, 1>))
                     : (vec ? run(state_runs_kernel<false, true, 2>) : run(state_runs_kernel<false, false, 2>));
}

// y: fp32 [T][width]; z: fp32 rows `z_stride` apart; weight: fp32 [width]; out: [T][width].  The width is cut into
// `groups` equal runs, each normed on its own.
FWB_API int fwb_gate_group_norm(const float* y, const float* z, long long z_stride, const float* weight, float eps,
                                void* out, int out_bf16, int T, int width, int groups, cudaStream_t stream) {
    if (T <= 0) return FWB_OK;
    if (!y || !z || !weight || !out || width <= 0 || groups <= 0 || width % groups || z_stride < width)
        return FWB_BAD_ARGUMENT;
    const int part = width / groups;
    const size_t smem = (size_t)part * sizeof(float);
    if (smem > 160 * 1024 || groups > 65535) return FWB_TOO_LARGE;
    auto launch = [&](auto kernel, auto rows) -> int {
        if (smem > 48 * 1024) {
            cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (err != cudaSuccess) return (int)err;
        }
        fwb::pdl(kernel, dim3(T, groups), part >= 1024 ? 256 : 128, smem, stream)(y, z, z_stride, weight, eps, rows, width, part);
        return fwb_launch_status();
    };
    return out_bf16 ? launch(gate_group_norm_kernel<__nv_bfloat16>, (__nv_bfloat16*)out)
                    : launch(gate_group_norm_kernel<float>, (float*)out);
}
