// Shared device helpers for the flyweight_b200 kernels (sm_100a only).
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define FWB_API extern "C" __attribute__((visibility("default")))

// Status codes returned by every host launcher.  0 = launched; a positive value
// is a cudaError_t from the launch; negative values are refusals made on the
// host before anything ran.
enum FwbStatus : int {
    FWB_OK = 0,
    FWB_BAD_ARGUMENT = -1,     // a size, stride or pointer the kernel cannot take
    FWB_UNSUPPORTED = -2,      // a combination the kernel was not written for
    FWB_TOO_LARGE = -3,        // beyond a stated maximum
};

static inline int fwb_launch_status() {
    cudaError_t err = cudaPeekAtLastError();
    return err == cudaSuccess ? FWB_OK : static_cast<int>(err);
}

namespace fwb {

// ---- programmatic dependent launch ------------------------------------------------
// Every kernel of the library is launched with programmatic stream serialisation: the next
// kernel in the stream may be scheduled while this one still runs, and does its set-up
// (shared-memory barriers, tensor-memory allocation, weight prefetch) in that shadow.
// pdl_wait() returns once the previous kernel has completed and its writes are visible; no
// kernel reads or writes anything another kernel touches before it.
__device__ __forceinline__ void pdl_launch_dependents() {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_entry() {
    pdl_launch_dependents();
    pdl_wait();
}

inline bool& pdl_enabled() {
    static bool enabled = true;
    return enabled;
}

template <typename Kernel>
struct PdlLauncher {
    Kernel kernel;
    dim3 grid, block;
    size_t smem;
    cudaStream_t stream;
    template <typename... Args>
    void operator()(Args... args) const {
        cudaLaunchConfig_t config = {};
        config.gridDim = grid;
        config.blockDim = block;
        config.dynamicSmemBytes = smem;
        config.stream = stream;
        cudaLaunchAttribute attr[1];
        attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[0].val.programmaticStreamSerializationAllowed = 1;
        config.attrs = attr;
        config.numAttrs = pdl_enabled() ? 1 : 0;
        cudaLaunchKernelEx(&config, kernel, args...);   // errors surface through fwb_launch_status()
    }
};
template <typename Kernel>
PdlLauncher<Kernel> pdl(Kernel kernel, dim3 grid, dim3 block, size_t smem, cudaStream_t stream) {
    return PdlLauncher<Kernel>{kernel, grid, block, smem, stream};
}

// ---- element access: everything is computed in fp32, stored as T --------------
template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) {
    return __bfloat162float(v);
}
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) {
    return __float2bfloat16_rn(v);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int offset = 16; offset > 0; offset >>= 1) v += __shfl_xor_sync(0xffffffffu, v, offset);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int offset = 16; offset > 0; offset >>= 1)
        v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, offset));
    return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result.  `scratch`
// holds 33 floats of shared memory.  The order of additions is fixed by the
// block size alone, so equal inputs give equal sums.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        const int warps = (blockDim.x + 31) >> 5;
        float t = lane < warps ? scratch[lane] : 0.0f;
        t = warp_sum(t);
        if (lane == 0) scratch[32] = t;
    }
    __syncthreads();
    return scratch[32];
}

// The lowest position a query at `pos` may see, from the one mask parameter every attention kernel
// takes.  span > 0: a sliding window, the last `span` positions up to pos.  span < 0: the sequence is
// cut into runs of -span positions counted from position 0, and a query sees only the keys of its own
// run (up to itself).  span == 0: every key from position 0 on.
__host__ __device__ __forceinline__ int first_visible_key(int pos, int span) {
    if (span > 0) return pos - span + 1 > 0 ? pos - span + 1 : 0;
    if (span < 0) return pos - pos % (-span);
    return 0;
}

// Which key tiles (of `tile` positions) a walk from the lowest visible key `lo` to `last` touches when the
// sequence's first `keep` positions stay visible beside a sliding window: `kept` tiles from position 0 on
// that end before the window's first tile, then the window's own.  keep == 0: the window's alone.
struct KeyTiles {
    int kept, first, count;      // tile i of `count`: i while i < kept, then first + (i - kept)
    __device__ __forceinline__ int at(int i) const { return i < kept ? i : first + (i - kept); }
};
__device__ __forceinline__ KeyTiles key_tiles(int lo, int last, int keep, int tile) {
    KeyTiles w;
    w.first = lo / tile;
    w.kept = (keep + tile - 1) / tile;
    if (w.kept > w.first) w.kept = w.first;
    w.count = w.kept + last / tile + 1 - w.first;
    return w;
}

// The tanh form of gelu: 0.5 g (1 + tanh(sqrt(2/pi) (g + 0.044715 g^3))).
__device__ __forceinline__ float gelu_tanh_f32(float g) {
    return 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
}

// silu(g) = g * sigmoid(g), sigmoid split by sign so neither branch overflows.
// tanh with an absolute error of a few 1e-8 from one fast exponential: (1 - e) / (1 + e), e = exp(-2|x|)
// (for the capped scores of the tensor-core attention kernels; the fp32 kernels call tanhf)
__device__ __forceinline__ float tanh_fast_f32(float x) {
    const float e = __expf(-2.0f * fabsf(x));
    return copysignf(__fdividef(1.0f - e, 1.0f + e), x);
}

// tanh for |x| <= TANH_SMALL without the special-function unit: the odd polynomial of degree 9 with the slope 1
// at 0 that is closest to it there in relative terms (least squares, reweighted until the error was level; 1.5e-8
// before rounding).  For capped scores, which rarely come near their cap.
constexpr float TANH_SMALL = 0.5f;
__device__ __forceinline__ float tanh_small_f32(float x) {
    const float y = x * x;
    const float q = fmaf(fmaf(fmaf(0.017241491f, y, -0.0530454926f), y, 0.13325879f), y, -0.333331436f);
    return fmaf(x * y, q, x);
}

__device__ __forceinline__ float silu_f32(float g) {
    const float e = expf(-fabsf(g));
    const float sig = g >= 0.0f ? 1.0f / (1.0f + e) : e / (1.0f + e);
    return g * sig;
}

// What a gated feed-forward makes of a gate value g and an up value u.  0: silu(g) u.  1: gelu(g) u (tanh
// form).  2, the clamped swish: g is cut off above `limit`, u is held inside [-limit, limit], and the
// result is g sigmoid(1.702 g) (u + 1).  3: max(g, 0) u.
constexpr int GATED_SILU = 0, GATED_GELU_TANH = 1, GATED_SWISH_CLAMPED = 2, GATED_RELU = 3;
constexpr float SWISH_CLAMPED_SLOPE = 1.702f;
__device__ __forceinline__ float gated_f32(int act, float limit, float g, float u) {
    if (act == GATED_SWISH_CLAMPED) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        const float z = SWISH_CLAMPED_SLOPE * g;
        const float e = expf(-fabsf(z));
        const float sig = z >= 0.0f ? 1.0f / (1.0f + e) : e / (1.0f + e);
        return g * sig * (u + 1.0f);
    }
    if (act == GATED_RELU) return fmaxf(g, 0.0f) * u;
    return (act == GATED_GELU_TANH ? gelu_tanh_f32(g) : silu_f32(g)) * u;
}

// What a product without a gate may do to its output before it is stored.  0: nothing.  1: max(v, 0)^2.
constexpr int OUTPUT_AS_IS = 0, OUTPUT_RELU_SQUARED = 1;
__device__ __forceinline__ float output_act_f32(int act, float v) {
    if (act != OUTPUT_RELU_SQUARED) return v;
    const float r = fmaxf(v, 0.0f);
    return r * r;
}

}  // namespace fwb
