// A residual of several streams.  A token carries S rows X_1 .. X_S of `hidden` 32-bit values ([token][stream][hidden]).
// A sublayer reads u = sum_s in[s] X_s, normed, and its result y goes back into every stream,
//
//   X_t <- sum_s mix[s][t] X_s + sum_j coef[j][t] y_j         (mix: [from][to]; all streams from the old ones)
//
// fx_stream_step does both ends in one pass over a token's rows: the update with up to three 32-bit results y_0 .. y_2
// and one that is still spread over the rows of the token's experts (y_3 = sum_k weight[k] rows[place[k]] + shared row),
// and then, on the new streams, what the next sublayer reads: x = rms(sum_t in[t] X_t) * w.  Without `mix` the streams
// stay as they are and u = sum_s in[s] X_s + sum_j coef[j][0] y_j: since in, mix and coef are known constants, what a
// sublayer in the middle of a layer reads can be had from the layer's old streams and the results so far, and the
// streams are written once a layer.  The constants travel as kernel arguments (the constant bank feeds the multiplies).
//
// One block a token; a thread takes four neighbouring elements of all streams at a time (one where rows are not whole
// 16-byte pieces).  u waits in shared memory for the sum of its squares.  All arithmetic is 32-bit.
#include "common.cuh"
#include "api.h"

namespace {

constexpr int MAX_S = FX_MAX_STREAMS;

template <int N> __device__ __forceinline__ void load32(const float* p, float* o) {
    if (N == 4) Pack<float>::load(p, o); else o[0] = *p;
}
template <int N> __device__ __forceinline__ void store32(float* p, const float* o) {
    if (N == 4) Pack<float>::store(p, o); else *p = o[0];
}
// N elements of a row whose type is known at run time
template <int N> __device__ __forceinline__ void load_row(const void* p, int dtype, long at, float* o) {
    if (dtype == FX_F32) { load32<N>(reinterpret_cast<const float*>(p) + at, o); return; }
    const bf16* b = reinterpret_cast<const bf16*>(p) + at;
    if (N == 1) { o[0] = to_f32(*b); return; }
    const uint2 v = *reinterpret_cast<const uint2*>(b);
    o[0] = __uint_as_float(v.x << 16); o[1] = __uint_as_float(v.x & 0xffff0000u);
    o[2] = __uint_as_float(v.y << 16); o[3] = __uint_as_float(v.y & 0xffff0000u);
}

// EXPERTS: 0 none, 1 any, 2 bfloat16 rows of at most MAX_K experts, whose loads are all on their way together with the
// streams'.
constexpr int MAX_K = 8;

template <int S, int N, int EXPERTS>
__global__ void __launch_bounds__(512) stream_step_kernel(const StreamStep a)
{
    extern __shared__ __align__(16) float u_s[];
    __shared__ float scratch[33];
    fx_pdl_wait();
    const int W = a.hidden;
    const long t = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
    float* X = a.streams + t * S * W;
    float sg = 1.f;
    if (a.shared && a.shared_gate) sg = 1.0f / (1.0f + expf(-a.shared_gate[t * a.gate_ld]));
    float ss = 0.f;
    long er[MAX_K];       // where the token's experts' rows start
    float ew[MAX_K];
    if (EXPERTS == 2) {
#pragma unroll
        for (int k = 0; k < MAX_K; ++k)
            if (k < a.top_k) {
                er[k] = (long)a.place[t * a.top_k + k] * W;
                ew[k] = a.weight ? a.weight[t * a.top_k + k] : 1.f;
            }
    }
    for (int i = threadIdx.x * N; i < W; i += blockDim.x * N) {
        float x[S][N], y[3][N], e[N];
        uint2 raw[MAX_K + 1];
        if (EXPERTS == 2) {
            const bf16* rows = reinterpret_cast<const bf16*>(a.expert_rows) + i;
#pragma unroll
            for (int k = 0; k < MAX_K; ++k)
                if (k < a.top_k) raw[k] = *reinterpret_cast<const uint2*>(rows + er[k]);
            if (a.shared) raw[MAX_K] = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(a.shared) + t * W + i);
        }
#pragma unroll
        for (int s = 0; s < S; ++s) load32<N>(X + (long)s * W + i, x[s]);
#pragma unroll
        for (int j = 0; j < 3; ++j)
            if (j < a.n_terms) load32<N>(a.y[j] + t * W + i, y[j]);
        if (EXPERTS == 2) {
            auto add = [&](uint2 r, float w) {      // (N is 4 here)
                e[0] = fmaf(w, __uint_as_float(r.x << 16), e[0]);
                e[N > 1 ? 1 : 0] = fmaf(w, __uint_as_float(r.x & 0xffff0000u), e[N > 1 ? 1 : 0]);
                e[N > 2 ? 2 : 0] = fmaf(w, __uint_as_float(r.y << 16), e[N > 2 ? 2 : 0]);
                e[N > 3 ? 3 : 0] = fmaf(w, __uint_as_float(r.y & 0xffff0000u), e[N > 3 ? 3 : 0]);
            };
#pragma unroll
            for (int n = 0; n < N; ++n) e[n] = 0.f;
#pragma unroll
            for (int k = 0; k < MAX_K; ++k)
                if (k < a.top_k) add(raw[k], ew[k]);
            if (a.shared) add(raw[MAX_K], sg);
        } else if (EXPERTS == 1) {
#pragma unroll
            for (int n = 0; n < N; ++n) e[n] = 0.f;
#pragma unroll 4
            for (int k = 0; k < a.top_k; ++k) {
                const long r = a.place[t * a.top_k + k];
                const float w = a.weight ? a.weight[t * a.top_k + k] : 1.f;
                float v[N];
                load_row<N>(a.expert_rows, a.expert_dtype, r * W + i, v);
#pragma unroll
                for (int n = 0; n < N; ++n) e[n] = fmaf(w, v[n], e[n]);
            }
            if (a.shared) {
                float v[N];
                load_row<N>(a.shared, a.expert_dtype, t * W + i, v);
#pragma unroll
                for (int n = 0; n < N; ++n) e[n] = fmaf(sg, v[n], e[n]);
            }
        }
        float u[N];
#pragma unroll
        for (int n = 0; n < N; ++n) u[n] = 0.f;
        if (a.write) {
#pragma unroll
            for (int to = 0; to < S; ++to) {
                float z[N];
#pragma unroll
                for (int n = 0; n < N; ++n) z[n] = 0.f;
#pragma unroll
                for (int s = 0; s < S; ++s)
#pragma unroll
                    for (int n = 0; n < N; ++n) z[n] = fmaf(a.mix[s][to], x[s][n], z[n]);
#pragma unroll
                for (int j = 0; j < 3; ++j)
                    if (j < a.n_terms) {
#pragma unroll
                        for (int n = 0; n < N; ++n) z[n] = fmaf(a.coef[j][to], y[j][n], z[n]);
                    }
                if (EXPERTS) {
#pragma unroll
                    for (int n = 0; n < N; ++n) z[n] = fmaf(a.coef[3][to], e[n], z[n]);
                }
                store32<N>(X + (long)to * W + i, z);
#pragma unroll
                for (int n = 0; n < N; ++n) u[n] = fmaf(a.in[to], z[n], u[n]);
            }
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s)
#pragma unroll
                for (int n = 0; n < N; ++n) u[n] = fmaf(a.in[s], x[s][n], u[n]);
#pragma unroll
            for (int j = 0; j < 3; ++j)
                if (j < a.n_terms) {
#pragma unroll
                    for (int n = 0; n < N; ++n) u[n] = fmaf(a.coef[j][0], y[j][n], u[n]);
                }
            if (EXPERTS) {
#pragma unroll
                for (int n = 0; n < N; ++n) u[n] = fmaf(a.coef[3][0], e[n], u[n]);
            }
        }
        if (a.x_out) {
            store32<N>(u_s + i, u);      // (read back by the same thread)
#pragma unroll
            for (int n = 0; n < N; ++n) ss = fmaf(u[n], u[n], ss);
        }
    }
    if (!a.x_out) return;      // (uniform)
    ss = block_sum(ss, scratch);
    const float r = 1.0f / sqrtf(ss / (float)W + a.eps);
    for (int i = threadIdx.x * N; i < W; i += blockDim.x * N) {
        float u[N], w[N];
        load32<N>(u_s + i, u);
        load_row<N>(a.w, a.w_dtype, i, w);
#pragma unroll
        for (int n = 0; n < N; ++n) u[n] = u[n] * r * w[n];
        const long at = (long)blockIdx.x * W + i;
        if (a.x_dtype == FX_F32) { store32<N>(reinterpret_cast<float*>(a.x_out) + at, u); continue; }
        bf16* o = reinterpret_cast<bf16*>(a.x_out) + at;
        if (N == 1) { *o = from_f32<bf16>(u[0]); continue; }
        __nv_bfloat162 p = __floats2bfloat162_rn(u[0], u[N > 1 ? 1 : 0]), q = __floats2bfloat162_rn(u[N > 1 ? 2 : 0], u[N > 1 ? 3 : 0]);
        *reinterpret_cast<uint2*>(o) = make_uint2(*reinterpret_cast<uint32_t*>(&p), *reinterpret_cast<uint32_t*>(&q));
    }
}

template <int S>
int launch(const StreamStep& a, int n_rows, bool vec, cudaStream_t s)
{
    const int items = vec ? a.hidden / 4 : a.hidden;
    // few rows (a decode step): a block's trips through its row are the kernel's time, so an item a thread
    const int most = n_rows >= 256 ? 256 : 512;
    int nt = 64;
    while (nt < items && nt < most) nt <<= 1;
    const size_t smem = a.x_out ? (size_t)((a.hidden + 3) & ~3) * 4 : 0;
    const bool ahead = vec && a.expert_dtype == FX_BF16 && a.top_k <= MAX_K;
    auto kern = a.place ? (ahead ? stream_step_kernel<S, 4, 2> : vec ? stream_step_kernel<S, 4, 1> : stream_step_kernel<S, 1, 1>)
                        : (vec ? stream_step_kernel<S, 4, 0> : stream_step_kernel<S, 1, 0>);
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    fx_launch_pdl(kern, n_rows, nt, smem, s, a);
    return fx_launch_status();
}

// S copies of every token's embedding row, times a constant.
template <typename T>
__global__ void embed_streams_kernel(const T* __restrict__ table, const int* __restrict__ ids, float* __restrict__ out,
                                     int hidden, int vocab, int streams, float scale, int* __restrict__ status)
{
    fx_pdl_wait();
    const long t = blockIdx.x;
    const int id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    if (!ok && threadIdx.x == 0 && status) atomicExch(status, 1);
    const T* row = table + (long)(ok ? id : 0) * hidden;
    float* o = out + t * streams * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = ok ? to_f32(row[i]) * scale : 0.f;
        for (int s = 0; s < streams; ++s) o[(long)s * hidden + i] = v;
    }
}

}  // namespace

extern "C" int fx_stream_step(const StreamStep* step, int n_streams, int n_rows, void* stream)
{
    if (n_rows <= 0) return FX_OK;
    const StreamStep& a = *step;
    if (a.hidden <= 0 || a.hidden > 50000 || n_streams < 1 || n_streams > MAX_S || a.n_terms < 0 || a.n_terms > 3 || !a.streams)
        return FX_ERR_SIZE;
    if ((a.place && (a.top_k <= 0 || !a.expert_rows)) || (a.shared && !a.place) || (a.x_out && !a.w) || (a.rows && a.write))
        return FX_ERR_SIZE;
    bool vec = a.hidden % 4 == 0;
    const void* p[] = {a.streams, a.y[0], a.y[1], a.y[2], a.expert_rows, a.shared, a.x_out, a.w};
    for (const void* q : p) vec = vec && (uintptr_t)q % 16 == 0;
    for (int j = 0; j < a.n_terms; ++j) if (!a.y[j]) return FX_ERR_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    switch (n_streams) {
        case 1: return launch<1>(a, n_rows, vec, s);
        case 2: return launch<2>(a, n_rows, vec, s);
        case 3: return launch<3>(a, n_rows, vec, s);
        case 4: return launch<4>(a, n_rows, vec, s);
        case 5: return launch<5>(a, n_rows, vec, s);
        case 6: return launch<6>(a, n_rows, vec, s);
        case 7: return launch<7>(a, n_rows, vec, s);
        default: return launch<8>(a, n_rows, vec, s);
    }
}

extern "C" int fx_embed_streams(const void* table, int dtype, const int* ids, float* out, int n_tokens, int hidden, int vocab,
                                int streams, float scale, int* status, void* stream)
{
    if (n_tokens <= 0) return FX_OK;
    if (hidden <= 0 || streams < 1) return FX_ERR_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    int nt = 32;
    while (nt < hidden && nt < 256) nt <<= 1;
    if (dtype == FX_F32) fx_launch_pdl(embed_streams_kernel<float>, n_tokens, nt, 0, s, (const float*)table, ids, out, hidden, vocab, streams, scale, status);
    else if (dtype == FX_BF16) fx_launch_pdl(embed_streams_kernel<bf16>, n_tokens, nt, 0, s, (const bf16*)table, ids, out, hidden, vocab, streams, scale, status);
    else return FX_ERR_DTYPE;
    return fx_launch_status();
}
