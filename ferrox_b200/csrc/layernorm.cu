// Layer norm (a weight, and a bias where the caller has one) over rows of the 32-bit residual stream, and the form
// that a block with norms on both sides of its sublayers needs: the sublayer's output is normed, added to the residual stream, and the new row is
// normed again for the sublayer that follows, in one pass over the row.
//
//   ln(z)[i] = (z[i] - mean(z)) / sqrt(mean((z - mean(z))^2) + eps) * w[i]
//
// All statistics are 32-bit, mean first and then the squared deviations (two passes: a difference of large sums
// would lose the small variances of a normed stream).  One block per row; a thread touches the same elements in
// every pass, so that a row may be normed in place and the second norm may read the row the first pass wrote.
#include "common.cuh"
#include "api.h"

namespace {

constexpr int LN_THREADS = 1024;   // at most; see ln_threads

struct RowStats { float mean, rstd; };

template <typename F>
__device__ __forceinline__ RowStats row_stats(F value, int n, float eps, float* scratch)
{
    float s = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) s += value(i);
    const float mean = block_sum(s, scratch) / (float)n;
    float d2 = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) { const float d = value(i) - mean; d2 = fmaf(d, d, d2); }
    const float var = block_sum(d2, scratch) / (float)n;
    return {mean, 1.0f / sqrtf(var + eps)};
}

template <typename OT>
__global__ void __launch_bounds__(LN_THREADS) layernorm_kernel(
    const float* x, const int* __restrict__ rows, const void* __restrict__ w, int w_dtype,
    const void* __restrict__ bias, int b_dtype, float eps, OT* out, int hidden)
{
    __shared__ float scratch[33];
    fx_pdl_wait();
    const int r = blockIdx.x;
    const float* xr = x + (long)(rows ? rows[r] : r) * hidden;
    const RowStats st = row_stats([&](int i) { return xr[i]; }, hidden, eps, scratch);
    OT* o = out + (long)r * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        float v = (xr[i] - st.mean) * st.rstd * load_any(w, w_dtype, i);
        if (bias) v += load_any(bias, b_dtype, i);
        o[i] = from_f32<OT>(v);
    }
}

// z = s1 * y1 (+ s2 * y2);  h += ln(z) * w_post;  x_out = ln(h) * w_next (if asked for).
template <typename OT>
__global__ void __launch_bounds__(LN_THREADS) layernorm_residual_kernel(
    float* h, const void* __restrict__ y1, int y1_dtype, float s1, const void* __restrict__ y2,
    int y2_dtype, float s2, const void* __restrict__ w_post, int wp_dtype, float eps, const void* __restrict__ w_next,
    int wn_dtype, float eps_next, OT* __restrict__ x_out, int hidden)
{
    __shared__ float scratch[33];
    fx_pdl_wait();
    const long base = (long)blockIdx.x * hidden;
    auto z = [&](int i) {
        float v = s1 * load_any(y1, y1_dtype, base + i);
        if (y2) v = fmaf(s2, load_any(y2, y2_dtype, base + i), v);
        return v;
    };
    const RowStats st = row_stats(z, hidden, eps, scratch);
    float* hr = h + base;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x)
        hr[i] = hr[i] + (z(i) - st.mean) * st.rstd * load_any(w_post, wp_dtype, i);
    if (!w_next) return;
    // the same thread wrote hr[i] that reads it here
    const RowStats sn = row_stats([&](int i) { return hr[i]; }, hidden, eps_next, scratch);
    OT* o = x_out + base;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x)
        o[i] = from_f32<OT>((hr[i] - sn.mean) * sn.rstd * load_any(w_next, wn_dtype, i));
}

// The RMS form: z = y, or z = sum_k weight[t, k] y[place[t, k]] (the rows of a token's experts, added up here) plus a
// shared expert's row;  h += z / sqrt(mean(z^2) + eps) * w_post;  x_out = h / sqrt(mean(h^2) + eps_next) * w_next (if
// asked for).  One block a row, which stays in registers from the first pass to the last: a thread holds up to CH items
// of N elements, N = 1 or 16 bytes of y.
template <typename T, int N> struct Row {
    static __device__ __forceinline__ void load(const T* p, float* o) { o[0] = to_f32(*p); }
};
template <> struct Row<float, 4> : Pack<float> {};
template <> struct Row<bf16, 8> : Pack<bf16> {};

constexpr int RMS_THREADS = 512;   // at most

// N weights of either element type (N > 1: 16-byte aligned vectors of them)
template <int N> __device__ __forceinline__ void load_weights(const void* w, int dtype, int i, float* o) {
    if (N == 1) { o[0] = load_any(w, dtype, i); return; }
    if (dtype == FX_F32) {
#pragma unroll
        for (int e = 0; e + 3 < N; e += 4) Pack<float>::load(reinterpret_cast<const float*>(w) + i + e, o + e);
    } else {
#pragma unroll
        for (int e = 0; e + 3 < N; e += 4) {
            const uint2 t = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(w) + i + e);
            o[e] = __uint_as_float(t.x << 16); o[e + 1] = __uint_as_float(t.x & 0xffff0000u);
            o[e + 2] = __uint_as_float(t.y << 16); o[e + 3] = __uint_as_float(t.y & 0xffff0000u);
        }
    }
}

struct RmsArgs {
    float* h; const void* y;
    const int* place; const float* weight; int top_k;         // place == nullptr: z is the token's own row of y
    const void* shared; const float* shared_gate; long gate_ld;
    const void* w_post; int wp_dtype; float eps;
    const void* w_next; int wn_dtype; float eps_next;         // w_next == nullptr: no second norm
    void* x_out; int hidden;
};

// EARLY (steps of few rows; CH = 1): a thread holds its weights from before the wait for the kernel before this one (which
// wrote none); with many rows the registers are worth more as blocks an SM holds.
template <typename T, typename OT, int N, int CH, bool EARLY>
__global__ void __launch_bounds__(RMS_THREADS, EARLY ? 1 : (N * CH <= 4 ? 3 : N * CH <= 16 ? 2 : 1)) rms_residual_kernel(RmsArgs a)
{
    __shared__ float scratch[33];
    float wp[N], wn[N];
    if (EARLY && (int)threadIdx.x * N < a.hidden) {
        load_weights<N>(a.w_post, a.wp_dtype, threadIdx.x * N, wp);
        if (a.w_next) load_weights<N>(a.w_next, a.wn_dtype, threadIdx.x * N, wn);
    }
    fx_pdl_wait();
    const int t = blockIdx.x;
    const T* y = reinterpret_cast<const T*>(a.y);
    const T* shared = reinterpret_cast<const T*>(a.shared);
    float* hr = a.h + (long)t * a.hidden;
    float sg = 1.f;
    if (shared && a.shared_gate) sg = 1.0f / (1.0f + expf(-a.shared_gate[(long)t * a.gate_ld]));
    float z[CH][N], hv[CH][N];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * blockDim.x + threadIdx.x) * N;
        if (i >= a.hidden) continue;
        // the stream's row is asked for together with y's
        if (N == 1) hv[c][0] = hr[i];
        else {
#pragma unroll
            for (int e = 0; e + 3 < N; e += 4) Pack<float>::load(hr + i + e, &hv[c][e]);
        }
        if (a.place) {
#pragma unroll
            for (int e = 0; e < N; ++e) z[c][e] = 0.f;
#pragma unroll 4
            for (int k = 0; k < a.top_k; ++k) {
                const long r = a.place[(long)t * a.top_k + k];
                const float w = a.weight ? a.weight[(long)t * a.top_k + k] : 1.f;
                float v[N];
                Row<T, N>::load(y + r * a.hidden + i, v);
#pragma unroll
                for (int e = 0; e < N; ++e) z[c][e] = fmaf(w, v[e], z[c][e]);
            }
            if (shared) {
                float v[N];
                Row<T, N>::load(shared + (long)t * a.hidden + i, v);
#pragma unroll
                for (int e = 0; e < N; ++e) z[c][e] = fmaf(sg, v[e], z[c][e]);
            }
        } else {
            Row<T, N>::load(y + (long)t * a.hidden + i, z[c]);
        }
#pragma unroll
        for (int e = 0; e < N; ++e) ss = fmaf(z[c][e], z[c][e], ss);
    }
    ss = block_sum(ss, scratch);
    const float r = 1.0f / sqrtf(ss / (float)a.hidden + a.eps);
    ss = 0.f;
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * blockDim.x + threadIdx.x) * N;
        if (i >= a.hidden) continue;
        if (!EARLY) load_weights<N>(a.w_post, a.wp_dtype, i, wp);
#pragma unroll
        for (int e = 0; e < N; ++e) {
            hv[c][e] += z[c][e] * r * wp[e];
            ss = fmaf(hv[c][e], hv[c][e], ss);
        }
        if (N == 1) hr[i] = hv[c][0];
        else {
#pragma unroll
            for (int e = 0; e + 3 < N; e += 4) Pack<float>::store(hr + i + e, &hv[c][e]);
        }
    }
    if (!a.w_next) return;      // (uniform)
    ss = block_sum(ss, scratch);
    const float rn = 1.0f / sqrtf(ss / (float)a.hidden + a.eps_next);
    OT* o = reinterpret_cast<OT*>(a.x_out) + (long)t * a.hidden;
#pragma unroll
    for (int c = 0; c < CH; ++c) {
        const int i = (c * blockDim.x + threadIdx.x) * N;
        if (i >= a.hidden) continue;
        if (!EARLY) load_weights<N>(a.w_next, a.wn_dtype, i, wn);
        float v[N];
#pragma unroll
        for (int e = 0; e < N; ++e) v[e] = hv[c][e] * rn * wn[e];
        if (N == 1) o[i] = from_f32<OT>(v[0]);
        else if (sizeof(OT) == 4) {
#pragma unroll
            for (int e = 0; e + 3 < N; e += 4) Pack<float>::store(reinterpret_cast<float*>(o) + i + e, v + e);
        } else {
#pragma unroll
            for (int e = 0; e + 1 < N; e += 2)
                *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<bf16*>(o) + i + e) = __floats2bfloat162_rn(v[e], v[e + 1]);
        }
    }
}

__global__ void scale_kernel(float* __restrict__ x, long n, float s)
{
    fx_pdl_wait();
    for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long)gridDim.x * blockDim.x) x[i] *= s;
}

// Few rows (a decode step) leave the kernel's time to the trips of one block through its row: more threads, fewer.
inline int ln_threads(int hidden, int n_rows)
{
    const int per = n_rows >= 256 ? 8 : 2;      // elements a thread; many rows fill the machine with smaller blocks
    int n = ((hidden + per - 1) / per + 31) / 32 * 32;
    return n < 64 ? 64 : (n > LN_THREADS ? LN_THREADS : n);
}

}  // namespace

extern "C" int fx_layernorm(const float* x, const int* rows, const void* w, int w_dtype, const void* bias, int b_dtype,
                            float eps, void* out, int out_dtype, int n_rows, int hidden, void* stream)
{
    if (n_rows <= 0) return FX_OK;
    if (hidden <= 0) return FX_ERR_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    if (out_dtype == FX_F32) fx_launch_pdl(layernorm_kernel<float>, n_rows, ln_threads(hidden, n_rows), 0, s, x, rows, w, w_dtype, bias, b_dtype, eps, (float*)out, hidden);
    else if (out_dtype == FX_BF16) fx_launch_pdl(layernorm_kernel<bf16>, n_rows, ln_threads(hidden, n_rows), 0, s, x, rows, w, w_dtype, bias, b_dtype, eps, (bf16*)out, hidden);
    else return FX_ERR_DTYPE;
    return fx_launch_status();
}

extern "C" int fx_layernorm_residual(float* h, const void* y1, int y1_dtype, float s1, const void* y2, int y2_dtype,
                                     float s2, const void* w_post, int wp_dtype, float eps, const void* w_next,
                                     int wn_dtype, float eps_next, void* x_out, int x_dtype, int n_rows, int hidden,
                                     void* stream)
{
    if (n_rows <= 0) return FX_OK;
    if (hidden <= 0 || !y1 || !w_post || (w_next && !x_out)) return FX_ERR_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    if (!w_next || x_dtype == FX_F32)
        fx_launch_pdl(layernorm_residual_kernel<float>, n_rows, ln_threads(hidden, n_rows), 0, s, h, y1, y1_dtype, s1, y2, y2_dtype, s2,
                      w_post, wp_dtype, eps, w_next, wn_dtype, eps_next, (float*)x_out, hidden);
    else if (x_dtype == FX_BF16)
        fx_launch_pdl(layernorm_residual_kernel<bf16>, n_rows, ln_threads(hidden, n_rows), 0, s, h, y1, y1_dtype, s1, y2, y2_dtype, s2,
                      w_post, wp_dtype, eps, w_next, wn_dtype, eps_next, (bf16*)x_out, hidden);
    else return FX_ERR_DTYPE;
    return fx_launch_status();
}

// h += rms(z) * w_post and, with w_next, x_out = rms(h) * w_next on the new rows; z as rms_residual_kernel says.  Refuses
// (FX_ERR_SIZE) rows of more than 16,384 elements (8,192 where rows are not 16-byte aligned).
extern "C" int fx_rmsnorm_residual(float* h, const void* y, int y_dtype, const int* place, const float* weight, int top_k,
                                   const void* shared, const float* shared_gate, long gate_ld, const void* w_post,
                                   int wp_dtype, float eps, const void* w_next, int wn_dtype, float eps_next, void* x_out,
                                   int x_dtype, int n_rows, int hidden, void* stream)
{
    if (n_rows <= 0) return FX_OK;
    if (hidden <= 0 || !y || !w_post || (w_next && !x_out) || (place && top_k <= 0) || (shared && !place)) return FX_ERR_SIZE;
    if ((y_dtype != FX_F32 && y_dtype != FX_BF16) || (w_next && x_dtype != FX_F32 && x_dtype != FX_BF16)) return FX_ERR_DTYPE;
    RmsArgs a;
    a.h = h; a.y = y; a.place = place; a.weight = weight; a.top_k = top_k; a.shared = shared; a.shared_gate = shared_gate;
    a.gate_ld = gate_ld; a.w_post = w_post; a.wp_dtype = wp_dtype; a.eps = eps; a.w_next = w_next; a.wn_dtype = wn_dtype;
    a.eps_next = eps_next; a.x_out = x_out; a.hidden = hidden;
    const int vw = y_dtype == FX_F32 ? 4 : 8;
    const bool vec = hidden % vw == 0 && (uintptr_t)h % 16 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)shared % 16 == 0 &&
                     (uintptr_t)x_out % 16 == 0 && (uintptr_t)w_post % 16 == 0 && (uintptr_t)w_next % 16 == 0;
    const int items = vec ? hidden / vw : hidden;
    // few rows (a decode step): a block's trips through its row are the kernel's time, so an item a thread
    int nt = 64;
    const int most = n_rows >= 256 ? 256 : RMS_THREADS, max_ch = vec ? 32 / vw : 16;
    while (nt < items && nt < most) nt <<= 1;
    while (fx_cdiv(items, nt) > max_ch && nt < RMS_THREADS) nt <<= 1;
    const int ch = (int)fx_cdiv(items, nt);
    if (ch > max_ch) return FX_ERR_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    const bool out32 = !w_next || x_dtype == FX_F32;
    const bool early = ch <= 1 && n_rows < 256;
#define FX_GO(T, OT, N, CH)                                                                                          \
    do { if (early) fx_launch_pdl(rms_residual_kernel<T, OT, N, CH, CH == 1>, n_rows, nt, 0, s, a);                 \
         else fx_launch_pdl(rms_residual_kernel<T, OT, N, CH, false>, n_rows, nt, 0, s, a); } while (0)
#define FX_CH(T, OT, N)                                                                                              \
    do { if (ch <= 1) FX_GO(T, OT, N, 1); else if (ch <= 2) FX_GO(T, OT, N, 2); else if (ch <= 4) FX_GO(T, OT, N, 4); \
         else if (ch <= 8) FX_GO(T, OT, N, (N == 8 ? 4 : 8)); else FX_GO(T, OT, N, (N == 1 ? 16 : 4)); } while (0)
    if (y_dtype == FX_F32) {
        if (vec) { if (out32) FX_CH(float, float, 4); else FX_CH(float, bf16, 4); }
        else { if (out32) FX_CH(float, float, 1); else FX_CH(float, bf16, 1); }
    } else {
        if (vec) { if (out32) FX_CH(bf16, float, 8); else FX_CH(bf16, bf16, 8); }
        else { if (out32) FX_CH(bf16, float, 1); else FX_CH(bf16, bf16, 1); }
    }
#undef FX_CH
#undef FX_GO
    return fx_launch_status();
}

extern "C" int fx_scale(float* x, long n, float scale, void* stream)
{
    if (n <= 0) return FX_OK;
    long blocks = fx_cdiv(n, 256);
    if (blocks > 4096) blocks = 4096;
    fx_launch_pdl(scale_kernel, (unsigned)blocks, 256, 0, (cudaStream_t)stream, x, n, scale);
    return fx_launch_status();
}
