// Head outputs on their way into an output product: packed side by side (without the zero channels that heads
// were padded with), turned back by the token's position where values were rotated, scaled, and written into
// columns of a row that other writers may share, so that one product takes the outputs of several mixers.
//
//   out[t][col0 + h e + c] = scale * turn(o[t][h][:], -position_t)[c]        c < e
//
// Behind the heads' columns up to col0 + width come `scale` split in two halves (value rounded to the row's
// type, and what the rounding left) and zeros: a product whose matrix holds a bias vector in those two
// columns adds scale * bias.
#include "common.cuh"

using namespace fwb;

namespace {

template <typename T>
__global__ void __launch_bounds__(256)
place_heads_kernel(const T* __restrict__ o, const int* __restrict__ positions, const float2* __restrict__ table,
                   int rot, int pairing, float scale, T* __restrict__ out, long long ld, int H, int D, int e,
                   int width) {
    fwb::pdl_entry();
    const int t = blockIdx.x;
    const T* src = o + (size_t)t * H * D;
    T* dst = out + (size_t)t * ld;
    const int half = rot / 2, rest = e - rot;
    const float2* cs = table ? table + (size_t)positions[t] * half : nullptr;
    for (int i = threadIdx.x; i < H * half; i += blockDim.x) {
        const int h = i / half, m = i - h * half;
        const int ia = pairing ? 2 * m : m, ib = pairing ? 2 * m + 1 : m + half;
        const float a = to_f32<T>(src[h * D + ia]), b = to_f32<T>(src[h * D + ib]);
        const float2 c = cs[m];
        dst[h * e + ia] = from_f32<T>((a * c.x + b * c.y) * scale);
        dst[h * e + ib] = from_f32<T>((b * c.x - a * c.y) * scale);
    }
    for (int i = threadIdx.x; i < H * rest; i += blockDim.x) {
        const int h = i / rest, c = rot + i - h * rest;
        dst[h * e + c] = from_f32<T>(to_f32<T>(src[h * D + c]) * scale);
    }
    for (int i = H * e + threadIdx.x; i < width; i += blockDim.x) {
        const int k = i - H * e;
        const T first = from_f32<T>(scale);
        dst[i] = k == 0 ? first : (k == 1 ? from_f32<T>(scale - to_f32<T>(first)) : from_f32<T>(0.0f));
    }
}

// bfloat16 heads in pieces of eight channels (16 bytes), interleaved pairs, whole head turned: D, e and the
// destination's columns are multiples of eight
__global__ void __launch_bounds__(256)
place_heads_bf16x8_kernel(const __nv_bfloat16* __restrict__ o, const int* __restrict__ positions,
                          const float4* __restrict__ table, int turned, float scale, __nv_bfloat16* __restrict__ out,
                          long long ld, int H, int D, int e, int width, int T) {
    fwb::pdl_entry();
    const int pieces = width >> 3, per_head = e >> 3;
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)T * pieces) return;
    const int t = (int)(i / pieces), piece = (int)(i - (size_t)t * pieces);
    __nv_bfloat162 r[4];
    if (piece < H * per_head) {
        const int h = piece / per_head, q = piece - h * per_head;
        const uint4 bits = *reinterpret_cast<const uint4*>(o + ((size_t)t * H + h) * D + 8 * q);
        const __nv_bfloat162* in = reinterpret_cast<const __nv_bfloat162*>(&bits);
        float4 c0 = make_float4(1.f, 0.f, 1.f, 0.f), c1 = c0;
        if (turned) {
            const float4* cs = table + (size_t)positions[t] * (e >> 2) + 2 * q;
            c0 = cs[0];
            c1 = cs[1];
        }
        const float co[4] = {c0.x, c0.z, c1.x, c1.z}, si[4] = {c0.y, c0.w, c1.y, c1.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 v = __bfloat1622float2(in[j]);
            r[j] = __floats2bfloat162_rn((v.x * co[j] + v.y * si[j]) * scale, (v.y * co[j] - v.x * si[j]) * scale);
        }
    } else {
        const __nv_bfloat16 first = __float2bfloat16_rn(scale), zero = __float2bfloat16_rn(0.0f);
        const __nv_bfloat16 left = __float2bfloat16_rn(scale - __bfloat162float(first));
        r[0] = piece == H * per_head ? __nv_bfloat162(first, left) : __nv_bfloat162(zero, zero);
#pragma unroll
        for (int j = 1; j < 4; ++j) r[j] = __nv_bfloat162(zero, zero);
    }
    *reinterpret_cast<uint4*>(out + (size_t)t * ld + 8 * piece) = *reinterpret_cast<const uint4*>(r);
}

}  // namespace

// o: [T][H][D], heads of D channels of which the first e count.  table: [positions][rot / 2] (cos, sin) or null
// (nothing turns); rot channels of a head turn back by table[positions[t]].  pairing 0 half-split, 1
// interleaved.  out: points at the first of the row's columns to write, rows `ld` entries apart; columns
// H e .. width - 1 hold the constant described above and zeros.  Both fp32 (bf16 0) or both bfloat16 (1).
FWB_API int fwb_place_heads(const void* o, const int* positions, const void* table, int rot, int pairing, float scale,
                            void* out, long long ld, int bf16, int T, int H, int D, int e, int width,
                            cudaStream_t stream) {
    if (T <= 0) return FWB_OK;
    if (!o || !out || H <= 0 || e <= 0 || D < e || width < H * e || ld < width) return FWB_BAD_ARGUMENT;
    if (!table) rot = 0;
    if (rot < 0 || rot > e || (rot & 1) || (rot && !positions) || (pairing != 0 && pairing != 1)) return FWB_BAD_ARGUMENT;
    using bf = __nv_bfloat16;
    if (bf16 && e % 8 == 0 && D % 8 == 0 && width % 8 == 0 && ld % 8 == 0 && (rot == 0 || (rot == e && pairing == 1)) &&
        (((uintptr_t)o | (uintptr_t)out | (uintptr_t)table) & 15) == 0) {
        const size_t pieces = (size_t)T * (width / 8);
        if (pieces / 256 > 2147483000) return FWB_TOO_LARGE;
        fwb::pdl(place_heads_bf16x8_kernel, (unsigned)((pieces + 255) / 256), 256, 0, stream)(
            (const bf*)o, positions, (const float4*)table, rot ? 1 : 0, scale, (bf*)out, ld, H, D, e, width, T);
        return fwb_launch_status();
    }
    if (bf16)
        fwb::pdl(place_heads_kernel<bf>, T, 256, 0, stream)((const bf*)o, positions, (const float2*)table, rot, pairing,
                                                            scale, (bf*)out, ld, H, D, e, width);
    else
        fwb::pdl(place_heads_kernel<float>, T, 256, 0, stream)((const float*)o, positions, (const float2*)table, rot,
                                                               pairing, scale, (float*)out, ld, H, D, e, width);
    return fwb_launch_status();
}
