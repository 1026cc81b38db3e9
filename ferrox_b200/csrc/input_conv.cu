// A causal convolution over time on every channel of a mixer's input, added to the input itself:
//
//   out[t, c] = x[t, c] + sum_j w[c, j] * x[t - (taps - 1) + j, c]        (zeros before the request's start)
//
// (add_input = 0: the sum alone, for a convolution that stands in its input's place, as the one behind the
// projections of an attention mixer; a bias per channel and SiLU of the result are options)
//
// over the tokens of one request.  The taps - 1 inputs before a step's first token come from the request's state
// slot (`tail` [slots, taps - 1, channels], 32-bit, oldest first), so a request may be cut into steps anywhere;
// after the step the last taps - 1 inputs of every entry become its tail (fx_conv_tail_update, linear_state.cu; a
// step of one token a request moves the tail on in this kernel).  The sum is 32-bit, taken in the order of the
// taps; the rows keep the element type of the mixer's input.
//
// Also here: the embedding with a learned position vector, the soft cap of the logits, the squared ReLU.
#include "common.cuh"
#include "api.h"

namespace {

constexpr int CONV_THREADS = 256;
constexpr int CONV_MAX_TAPS = 16;

template <typename T>
__global__ void __launch_bounds__(CONV_THREADS) input_conv_kernel(
    const T* __restrict__ x, long ldx, const void* __restrict__ w, int w_dtype, int taps, float* tail,
    const int* __restrict__ token_seq, const int* __restrict__ seq_slot, T* __restrict__ out, long ldo, int C,
    int update_tail, int add_input, const void* __restrict__ bias, int b_dtype, int act)
{
    fx_pdl_wait();
    const int t = blockIdx.x;
    const int c = blockIdx.y * CONV_THREADS + threadIdx.x;
    if (c >= C) return;
    const int b = token_seq[t];
    // how many rows before t belong to the same entry (at most taps - 1 matter)
    int own = 0;
    while (own < taps - 1 && t - own - 1 >= 0 && token_seq[t - own - 1] == b) ++own;
    float* tl = tail + (long)seq_slot[b] * (taps - 1) * C;
    const float xt = to_f32(x[(long)t * ldx + c]);
    float acc = add_input ? xt : 0.f;     // (a convolution that replaces its input: the sum alone)
    if (bias) acc += load_any(bias, b_dtype, c);
    for (int j = 0; j < taps; ++j) {
        const int back = taps - 1 - j;          // this tap's input lies `back` tokens before t
        float v;
        if (back == 0) v = xt;
        else if (back <= own) v = to_f32(x[(long)(t - back) * ldx + c]);
        else v = tl[(long)(taps - 1 - (back - own)) * C + c];
        acc = fmaf(load_any(w, w_dtype, (long)c * taps + j), v, acc);
    }
    if (act) acc = acc / (1.0f + expf(-acc));
    out[(long)t * ldo + c] = from_f32<T>(acc);
    // (the caller's promise that every entry brings exactly one token: this thread is then the only reader of the
    // channel's tail in the whole step, and moves it on by the token's input itself)
    if (update_tail && taps > 1) {
        for (int j = 0; j + 1 < taps - 1; ++j) tl[(long)j * C + c] = tl[(long)(j + 1) * C + c];
        tl[(long)(taps - 2) * C + c] = xt;
    }
}

// The same for a prompt: a thread takes RUN tokens of two neighbouring channels one after the other and keeps the last
// TAPS - 1 inputs in registers, so that every input is read once (and TAPS - 1 more at the start of a run).
constexpr int CONV_RUN = 16;

template <typename T> __device__ __forceinline__ float2 load2(const T* p);
template <> __device__ __forceinline__ float2 load2<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <> __device__ __forceinline__ float2 load2<bf16>(const bf16* p) {
    return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
template <typename T> struct T2;      // two neighbouring elements as they lie in memory
template <> struct T2<float> {
    float2 v;
    __device__ __forceinline__ void load(const float* p) { v = *reinterpret_cast<const float2*>(p); }
    __device__ __forceinline__ float2 value() const { return v; }
};
template <> struct T2<bf16> {
    __nv_bfloat162 v;
    __device__ __forceinline__ void load(const bf16* p) { v = *reinterpret_cast<const __nv_bfloat162*>(p); }
    __device__ __forceinline__ float2 value() const { return __bfloat1622float2(v); }
};
__device__ __forceinline__ void store2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void store2(bf16* p, float2 v) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y);
}

template <typename T, int TAPS>
__global__ void __launch_bounds__(CONV_THREADS) input_conv_run_kernel(
    const T* __restrict__ x, long ldx, const void* __restrict__ w, int w_dtype, const float* __restrict__ tail,
    const int* __restrict__ token_seq, const int* __restrict__ seq_slot, T* __restrict__ out, long ldo, int n_tokens, int C,
    int add_input, const void* __restrict__ bias, int b_dtype, int act)
{
    fx_pdl_wait();
    const int t0 = blockIdx.x * CONV_RUN, t1 = min(n_tokens, t0 + CONV_RUN);
    const int c = (blockIdx.y * CONV_THREADS + threadIdx.x) * 2;
    if (c >= C) return;
    float2 wt[TAPS], hist[TAPS];      // hist[j]: the input TAPS - 1 - j tokens before the current one
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
        wt[j] = make_float2(load_any(w, w_dtype, (long)c * TAPS + j), load_any(w, w_dtype, (long)(c + 1) * TAPS + j));
    float2 b0 = make_float2(0.f, 0.f);
    if (bias) b0 = make_float2(load_any(bias, b_dtype, c), load_any(bias, b_dtype, c + 1));
    // the run's inputs and entries, all asked for before the first is used
    T2<T> xs[CONV_RUN];
    int ss[CONV_RUN];
#pragma unroll
    for (int r = 0; r < CONV_RUN; ++r) {
        const int t = min(t0 + r, n_tokens - 1);
        xs[r].load(x + (long)t * ldx + c);
        ss[r] = token_seq[t];
    }
    int seq = -1;
#pragma unroll
    for (int r = 0; r < CONV_RUN; ++r) {
        const int t = t0 + r, s = ss[r];
        if (t >= t1) break;
        if (s != seq) {       // the run's first token, or another entry's: its earlier inputs, from rows and tail
            seq = s;
            int own = 0;
            while (own < TAPS - 1 && t - own - 1 >= 0 && token_seq[t - own - 1] == s) ++own;
            const float* tl = tail + (long)seq_slot[s] * (TAPS - 1) * C + c;
#pragma unroll
            for (int j = 1; j < TAPS; ++j) {            // (moved down by one below)
                const int back = TAPS - j;
                hist[j] = back <= own ? load2(x + (long)(t - back) * ldx + c)
                                      : *reinterpret_cast<const float2*>(tl + (long)(TAPS - 1 - (back - own)) * C);
            }
        }
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j) hist[j] = hist[j + 1];
        const float2 xt = xs[r].value();
        hist[TAPS - 1] = xt;
        float2 acc = add_input ? xt : make_float2(0.f, 0.f);
        acc.x += b0.x; acc.y += b0.y;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) { acc.x = fmaf(wt[j].x, hist[j].x, acc.x); acc.y = fmaf(wt[j].y, hist[j].y, acc.y); }
        if (act) { acc.x = acc.x / (1.0f + expf(-acc.x)); acc.y = acc.y / (1.0f + expf(-acc.y)); }
        store2(out + (long)t * ldo + c, acc);
    }
}

template <typename T, typename PT>
__global__ void embed_pos_kernel(const T* __restrict__ table, const int* __restrict__ ids, const PT* __restrict__ pos_table,
                                 const int* __restrict__ positions, float* __restrict__ out, int hidden, int vocab,
                                 int n_positions, int* __restrict__ status)
{
    fx_pdl_wait();
    const int t = blockIdx.x;
    const int id = ids[t], p = positions[t];
    const bool ok = id >= 0 && id < vocab, pok = p >= 0 && p < n_positions;
    if (threadIdx.x == 0 && status) {
        if (!ok) atomicExch(status, 1);
        else if (!pok) atomicExch(status, 4);
    }
    const T* row = table + (long)(ok ? id : 0) * hidden;
    const PT* prow = pos_table + (long)(pok ? p : 0) * hidden;
    float* o = out + (long)t * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x)
        o[i] = (ok && pok) ? to_f32(row[i]) + to_f32(prow[i]) : 0.f;
}

__global__ void softcap_kernel(float* __restrict__ x, long n, float cap)
{
    fx_pdl_wait();
    const float inv = 1.0f / cap;
    for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long)gridDim.x * blockDim.x)
        x[i] = cap * tanhf(x[i] * inv);
}

template <typename T>
__global__ void relu_square_kernel(T* __restrict__ x, long ld, int n)
{
    fx_pdl_wait();
    T* r = x + (long)blockIdx.x * ld;
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < n; i += gridDim.y * blockDim.x) {
        const float v = fmaxf(to_f32(r[i]), 0.f);
        r[i] = from_f32<T>(v * v);
    }
}

}  // namespace

extern "C" int fx_input_conv(const void* x, int dtype, long ldx, const void* w, int w_dtype, int taps, float* tail,
                             const int* token_seq, const int* seq_slot, void* out, long ldo, int n_tokens, int channels,
                             int update_tail, int add_input, const void* bias, int b_dtype, int act, void* stream)
{
    if (n_tokens <= 0 || channels <= 0) return FX_OK;
    if (taps < 1 || taps > CONV_MAX_TAPS || x == out) return FX_ERR_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    dim3 grid(n_tokens, (unsigned)fx_cdiv(channels, CONV_THREADS));
    const int es = dtype == FX_F32 ? 8 : 4;      // bytes of two elements
    if (!update_tail && n_tokens >= 128 && (taps == 3 || taps == 4) && channels % 2 == 0 && ldx % 2 == 0 && ldo % 2 == 0 &&
        (uintptr_t)x % es == 0 && (uintptr_t)out % es == 0 && (uintptr_t)tail % 8 == 0) {
        dim3 g((unsigned)fx_cdiv(n_tokens, CONV_RUN), (unsigned)fx_cdiv(channels, 2 * CONV_THREADS));
#define FX_RUN(T, TAPS)                                                                                              \
    fx_launch_pdl(input_conv_run_kernel<T, TAPS>, g, CONV_THREADS, 0, s, (const T*)x, ldx, w, w_dtype,               \
                  (const float*)tail, token_seq, seq_slot, (T*)out, ldo, n_tokens, channels, add_input, bias, b_dtype, act)
        if (dtype == FX_F32) { if (taps == 4) FX_RUN(float, 4); else FX_RUN(float, 3); }
        else if (dtype == FX_BF16) { if (taps == 4) FX_RUN(bf16, 4); else FX_RUN(bf16, 3); }
        else return FX_ERR_DTYPE;
#undef FX_RUN
        return fx_launch_status();
    }
    if (dtype == FX_F32)
        fx_launch_pdl(input_conv_kernel<float>, grid, CONV_THREADS, 0, s, (const float*)x, ldx, w, w_dtype, taps, tail,
                      token_seq, seq_slot, (float*)out, ldo, channels, update_tail, add_input, bias, b_dtype, act);
    else if (dtype == FX_BF16)
        fx_launch_pdl(input_conv_kernel<bf16>, grid, CONV_THREADS, 0, s, (const bf16*)x, ldx, w, w_dtype, taps, tail,
                      token_seq, seq_slot, (bf16*)out, ldo, channels, update_tail, add_input, bias, b_dtype, act);
    else return FX_ERR_DTYPE;
    return fx_launch_status();
}

extern "C" int fx_embed_pos(const void* table, int dtype, const int* ids, const void* pos_table, int pos_dtype,
                            const int* positions, float* out, int n_tokens, int hidden, int vocab, int n_positions,
                            int* status, void* stream)
{
    if (n_tokens <= 0) return FX_OK;
    cudaStream_t s = (cudaStream_t)stream;
    int nt = 32;
    while (nt < hidden && nt < 256) nt <<= 1;
#define FX_GO(T, PT)                                                                                                \
    fx_launch_pdl(embed_pos_kernel<T, PT>, n_tokens, nt, 0, s, (const T*)table, ids, (const PT*)pos_table, positions, \
                  out, hidden, vocab, n_positions, status)
    if (dtype == FX_F32 && pos_dtype == FX_F32) FX_GO(float, float);
    else if (dtype == FX_BF16 && pos_dtype == FX_BF16) FX_GO(bf16, bf16);
    else if (dtype == FX_F32 && pos_dtype == FX_BF16) FX_GO(float, bf16);
    else if (dtype == FX_BF16 && pos_dtype == FX_F32) FX_GO(bf16, float);
    else return FX_ERR_DTYPE;
#undef FX_GO
    return fx_launch_status();
}

extern "C" int fx_softcap(float* x, long n, float cap, void* stream)
{
    if (n <= 0) return FX_OK;
    if (!(cap > 0.f)) return FX_ERR_SIZE;
    long blocks = fx_cdiv(n, 256);
    if (blocks > 4096) blocks = 4096;
    fx_launch_pdl(softcap_kernel, (unsigned)blocks, 256, 0, (cudaStream_t)stream, x, n, cap);
    return fx_launch_status();
}

extern "C" int fx_relu_square(void* x, int dtype, long ld, int rows, int n, void* stream)
{
    if (rows <= 0 || n <= 0) return FX_OK;
    cudaStream_t s = (cudaStream_t)stream;
    long by = fx_cdiv(n, 256 * 4);
    if (by > 64) by = 64;
    dim3 grid(rows, (unsigned)by);
    if (dtype == FX_F32) fx_launch_pdl(relu_square_kernel<float>, grid, 256, 0, s, (float*)x, ld, n);
    else if (dtype == FX_BF16) fx_launch_pdl(relu_square_kernel<bf16>, grid, 256, 0, s, (bf16*)x, ld, n);
    else return FX_ERR_DTYPE;
    return fx_launch_status();
}
