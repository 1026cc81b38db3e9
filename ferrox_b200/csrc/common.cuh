// Shared helpers of the sm_100a kernels: element types, conversions, reductions,
// the status codes that the C entry points return.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

// Element type codes of the C ABI (ferrox_b200/kernels/lib.py mirrors them).
#define FX_F32 0
#define FX_BF16 1

// Status codes returned by every entry point. 0 = launched; positive values are
// cudaError_t from the launch; negative values are refusals of this library.
#define FX_OK 0
#define FX_ERR_DTYPE -1     // combination of element types not built
#define FX_ERR_SIZE -2      // a size outside what the kernel handles
#define FX_ERR_ALIGN -3     // pointer or stride not aligned as required
#define FX_ERR_TIMEOUT -4   // a bounded wait inside a kernel ran out

typedef __nv_bfloat16 bf16;

template <typename T> struct fx_code;
template <> struct fx_code<float> { static constexpr int value = FX_F32; };
template <> struct fx_code<bf16> { static constexpr int value = FX_BF16; };

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

// Read element i of an array whose element type is only known at run time
// (small tensors that keep their stored precision: norm weights, biases).
__device__ __forceinline__ float load_any(const void* p, int dtype, long i) {
    return dtype == FX_F32 ? reinterpret_cast<const float*>(p)[i]
                           : __bfloat162float(reinterpret_cast<const bf16*>(p)[i]);
}

// 16 bytes of a row as 32-bit values.
template <typename T> struct Pack;
template <> struct Pack<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void load(const float* p, float* o) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
    }
    static __device__ __forceinline__ void store(float* p, const float* o) {
        *reinterpret_cast<float4*>(p) = make_float4(o[0], o[1], o[2], o[3]);
    }
};
template <> struct Pack<bf16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void load(const bf16* p, float* o) {
        const uint4 v = *reinterpret_cast<const uint4*>(p);
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            o[2 * i] = __uint_as_float(w[i] << 16);
            o[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
    static __device__ __forceinline__ void store(bf16* p, const float* o) {
        uint4 v;
        __nv_bfloat162 a = __floats2bfloat162_rn(o[0], o[1]), b = __floats2bfloat162_rn(o[2], o[3]);
        __nv_bfloat162 c = __floats2bfloat162_rn(o[4], o[5]), d = __floats2bfloat162_rn(o[6], o[7]);
        v.x = *reinterpret_cast<uint32_t*>(&a); v.y = *reinterpret_cast<uint32_t*>(&b);
        v.z = *reinterpret_cast<uint32_t*>(&c); v.w = *reinterpret_cast<uint32_t*>(&d);
        *reinterpret_cast<uint4*>(p) = v;
    }
};

// What a plain product's result may pass through before it is stored (the kernels' `gated` argument below zero:
// -code): 1 the square of ReLU.
__device__ __forceinline__ float fx_unary(float x, int code) {
    if (code == 1) { x = fmaxf(x, 0.f); x *= x; }
    return x;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result. The order
// of additions is fixed by the thread layout alone.
__device__ __forceinline__ float block_sum(float v, float* scratch /* >= 33 floats */) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarp = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();  // scratch may still be read from an earlier call
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < nwarp ? scratch[lane] : 0.f;
        t = warp_sum(t);
        if (lane == 0) scratch[32] = t;
    }
    __syncthreads();
    return scratch[32];
}

// The clamped gated unit of a feed-forward: the gate is capped from above, the up value from both sides, the gate
// passes through g * sigmoid(alpha g) and multiplies (up + 1).  FAST: the hardware's exponential.
template <bool FAST>
__device__ __forceinline__ float fx_clamped_glu(float g, float u, float limit, float alpha) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return (FAST ? __fdividef(g, 1.0f + __expf(-alpha * g)) : g / (1.0f + expf(-alpha * g))) * (u + 1.0f);
}

// z * (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))) / 2, the tanh form of GELU, written with 1 + tanh(y) = 2 / (1 + e^(-2y)).
template <bool FAST>
__device__ __forceinline__ float fx_gelu_tanh(float z) {
    const float y2 = 1.5957691216057308f * fmaf(0.044715f * z * z, z, z);      // 2 sqrt(2/pi) (z + 0.044715 z^3)
    return FAST ? __fdividef(z, 1.0f + __expf(-y2)) : z / (1.0f + expf(-y2));
}

// A gated feed-forward's unit act(g) * u; act 0: SiLU, 1: ReLU, 2: the clamped unit, 3: GELU in its tanh form.  FAST:
// the hardware's exponential and quotient.
template <bool FAST>
__device__ __forceinline__ float fx_gate(float g, float u, int act, float limit, float alpha) {
    if (act == 2) return fx_clamped_glu<FAST>(g, u, limit, alpha);
    if (act == 1) return fmaxf(g, 0.f) * u;
    if (act == 3) return fx_gelu_tanh<FAST>(g) * u;
    return (FAST ? __fdividef(g, 1.0f + __expf(-g)) : g / (1.0f + expf(-g))) * u;
}

// The same over 32 pairs in registers, the choice of the unit made once: x[j] <- act(x[j]) * u[j].
__device__ __forceinline__ void fx_gate_32(float* x, const uint32_t* u, int act, float limit, float alpha) {
    if (act == 2) {
#pragma unroll
        for (int j = 0; j < 32; ++j) x[j] = fx_clamped_glu<true>(x[j], __uint_as_float(u[j]), limit, alpha);
    } else if (act == 0) {
#pragma unroll
        for (int j = 0; j < 32; ++j) x[j] = __fdividef(x[j], 1.0f + __expf(-x[j])) * __uint_as_float(u[j]);
    } else if (act == 1) {
#pragma unroll
        for (int j = 0; j < 32; ++j) x[j] = fmaxf(x[j], 0.f) * __uint_as_float(u[j]);
    } else {
#pragma unroll
        for (int j = 0; j < 32; ++j) x[j] = fx_gelu_tanh<true>(x[j]) * __uint_as_float(u[j]);
    }
}

// log(1 + e^x) = max(x, 0) + log(1 + e) with e = e^-|x| in (0, 1]; log(1 + e) = 2 artanh(s), s = e / (2 + e) <= 1/3, by
// its series 2 (s + s^3/3 + s^5/5 + ...), the first term left out below 2e-8 of the sum.
__device__ __forceinline__ float fx_softplus(float x)
{
    const float e = expf(-fabsf(x));
    const float s = e / (2.0f + e), s2 = s * s;
    float p = fmaf(s2, 1.0f / 15.0f, 1.0f / 13.0f);
    p = fmaf(p, s2, 1.0f / 11.0f);
    p = fmaf(p, s2, 1.0f / 9.0f);
    p = fmaf(p, s2, 1.0f / 7.0f);
    p = fmaf(p, s2, 1.0f / 5.0f);
    p = fmaf(p, s2, 1.0f / 3.0f);
    return fmaxf(x, 0.f) + 2.0f * fmaf(s * s2, p, s);
}

// sigmoid(g) with the hardware's exponential and quotient, for the attention kernels' output gates.
__device__ __forceinline__ float fx_sigmoid_fast(float g) { return __fdividef(1.0f, 1.0f + __expf(-g)); }

// A head's result turned back: pair (x0, x1) of neighbours 2m, 2m + 1 by minus the angle whose cos and sin are cs, for
// attention whose values were turned by their own positions before they were cached.
__device__ __forceinline__ void fx_turn_back(float& x0, float& x1, float2 cs) {
    const float a = x0;
    x0 = a * cs.x + x1 * cs.y;
    x1 = x1 * cs.x - a * cs.y;
}

// The same where the two elements of a pair lie in neighbouring lanes (even lane: x0): called by whole warps.
__device__ __forceinline__ float fx_turn_back_lane(float x, float2 cs, bool odd) {
    const float other = __shfl_xor_sync(0xffffffffu, x, 1);
    return odd ? x * cs.x - other * cs.y : x * cs.x + other * cs.y;
}

// The first key the query at position pos may see: of a window of the last `window` positions (0: no window) and of
// chunks of `chunk` positions counted from the request's start (0: no chunks), in which a query sees its own chunk only.
__host__ __device__ __forceinline__ int fx_first_key(int pos, int window, int chunk) {
    int lo = window > 0 && pos - window + 1 > 0 ? pos - window + 1 : 0;
    if (chunk > 0) { const int c = pos - pos % chunk; lo = c > lo ? c : lo; }
    return lo;
}

// Key range [k_begin, k_end) of run `split` of a decoding token at position pos whose first visible key is lo.
// split_len > 0: runs of split_len keys counted from position 0.  split_len == 0: the token's own visible keys,
// counted from the multiple of 64 at or below lo, cut into n_splits runs of equal length (a multiple of 64), so
// that every run has work whatever the context length is.  An empty range (k_begin >= k_end) has no block
// result and is skipped when the runs are merged.
__device__ __forceinline__ void fx_split_range(int pos, int lo, int split, int n_splits, int split_len, int& k_begin,
                                               int& k_end) {
    int base = 0, len = split_len;
    if (split_len <= 0) {
        base = lo & ~63;
        len = (((pos + 1 - base) + n_splits - 1) / n_splits + 63) & ~63;
    }
    k_begin = max(lo, base + split * len);
    k_end = min(pos + 1, base + (split + 1) * len);
}

// Programmatic dependent launch.  A kernel launched with fx_launch_pdl may be set up
// on the GPU while the kernel before it on the stream is still running; it must
// call fx_pdl_wait() before it touches anything that kernel wrote (here: first
// thing), which also lets the kernel after it start its own set-up.  Launch
// latencies of a chain of short kernels then overlap instead of adding up.
__device__ __forceinline__ void fx_pdl_wait() {
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}

// What may be read before the wait: constants, and with fx_ld_old what an earlier kernel or copy than the one before this
// one has written.  (A plain load may find a line in the SM's own cache that was read before it was written, when no kernel
// has come to its wait on this SM since: fx_ld_old asks the L2.)
__device__ __forceinline__ int fx_ld_old(const int* p) { return __ldcg(p); }

// The two halves apart, for a kernel that runs long on few warps (a recurrence over a prompt's tokens): it waits first
// thing and lets its dependents be set up when its long loop is over, so that their waiting blocks do not sit on its
// SMs meanwhile.
__device__ __forceinline__ void fx_pdl_wait_only() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void fx_pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

// fx_set_pdl(0) (elementwise.cu) makes fx_launch_pdl launch without the attribute; for measurements.
extern int g_fx_pdl_enabled;

template <typename... KArgs, typename... Args>
static inline void fx_launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                 Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = g_fx_pdl_enabled ? 1 : 0;
    cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);   // errors surface through cudaGetLastError
}

// The same launch with the early set-up left out when `early` is false.  For a kernel that runs long on few blocks (a
// recurrence over a prompt): blocks that are set up while the kernel before them still fills the device land where its
// blocks happen to end first, several on one SM beside SMs that get none, and stay there (a recurrence of 128 blocks
// over 2,048 tokens on a B200: 1.4 ms set up early, 0.65 ms on an empty device).  Its griddepcontrol instructions
// then do nothing, and the kernel after it may still be set up early.
template <typename... KArgs, typename... Args>
static inline void fx_launch_pdl_if(bool early, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                    cudaStream_t stream, Args... args) {
    if (early) { fx_launch_pdl(kernel, grid, block, smem, stream, args...); return; }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

static inline int fx_launch_status() {
    cudaError_t e = cudaGetLastError();
    return e == cudaSuccess ? FX_OK : (int)e;
}

static inline long fx_cdiv(long a, long b) { return (a + b - 1) / b; }

// Streaming multiprocessors of the current device, asked once (elementwise.cu); grids are sized by it.
extern "C" int fx_sm_count();
