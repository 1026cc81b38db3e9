// What stands between an attention mixer's projections and its attention kernel, for the mixers that do more
// there than rotate: queries and keys normed per head, a query temperature that grows with the position, keys
// and values of different widths; and the latent form, in which a position stores one normed latent vector and one
// rotated key part that all heads share.  All norms, angles, rotations and temperatures are 32-bit arithmetic;
// the rows keep the element type of the projections.
#include "common.cuh"
#include "api.h"

namespace {

// ---------------------------------------------------------------------------------------------------------------
// Rows of [q heads | k heads | v heads] (head widths D, D, V).  Per head, in place:
//   q <- q / sqrt(mean(q^2) + eps) * wq * (1 + coef * ln(floor((pos + 1) / every) + 1))
//   k <- k / sqrt(mean(k^2) + eps) * wk                      (wq, wk: [D], shared by the heads; null: no norm)
// then k and v go to the pages, [page][kv head][position][D] and [page][kv head][position][V].
// v_eps >= 0: every value head is divided by its root mean square first, v / sqrt(mean(v^2) + v_eps), no weight,
// and is cached so.
// One block a token, a warp a head.
template <typename T>
__global__ void qk_norm_store_kernel(T* __restrict__ qkv, long ld, const int* __restrict__ positions,
                                     const int* __restrict__ token_seq, const int* __restrict__ seq_slot,
                                     const void* __restrict__ wq, const void* __restrict__ wk, int w_dtype, float eps,
                                     float temp_coef, int temp_every, T* __restrict__ k_pages, T* __restrict__ v_pages,
                                     const int* __restrict__ block_table, int table_width, int page_size, int H, int G,
                                     int D, int V, int write_cache, int* __restrict__ status, float v_eps)
{
    fx_pdl_wait();
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const int pos = positions[t];
    T* row = qkv + (long)t * ld;
    long place = -1;      // (page, kv head 0, position in the page) as one index
    if (write_cache) {
        const int page = block_table[(long)seq_slot[token_seq[t]] * table_width + pos / page_size];
        if (page < 0) { if (threadIdx.x == 0 && status) atomicExch(status, 2); }
        else place = (long)page * G * page_size + (pos % page_size);
    }
    float temp = 1.f;
    if (temp_every > 0) temp = 1.0f + temp_coef * logf((float)((pos + 1) / temp_every + 1));
    for (int u = warp; u < H + G; u += n_warps) {
        const bool is_q = u < H;
        T* x = row + (long)u * D;
        const void* w = is_q ? wq : wk;
        float r = 1.f;
        if (w) {
            float ss = 0.f;
            for (int i = lane; i < D; i += 32) { const float v = to_f32(x[i]); ss = fmaf(v, v, ss); }
            ss = warp_sum(ss);
            r = sqrtf(ss / (float)D + eps);
        }
        const float mult = is_q ? temp : 1.f;
        T* kp = (!is_q && place >= 0) ? k_pages + (place + (long)(u - H) * page_size) * D : nullptr;
        for (int i = lane; i < D; i += 32) {
            float v = to_f32(x[i]);
            if (w) v = v / r * load_any(w, w_dtype, i);
            const T o = from_f32<T>(v * mult);
            x[i] = o;
            if (kp) kp[i] = o;
        }
    }
    if (place < 0) return;
    const T* v = row + (long)(H + G) * D;
    if (v_eps >= 0.f) {
        for (int g = warp; g < G; g += n_warps) {
            const T* x = v + (long)g * V;
            float ss = 0.f;
            for (int i = lane; i < V; i += 32) { const float f = to_f32(x[i]); ss = fmaf(f, f, ss); }
            ss = warp_sum(ss);
            const float r = sqrtf(ss / (float)V + v_eps);
            T* vp = v_pages + (place + (long)g * page_size) * V;
            for (int i = lane; i < V; i += 32) vp[i] = from_f32<T>(to_f32(x[i]) / r);
        }
        return;
    }
    for (int idx = threadIdx.x; idx < G * V; idx += blockDim.x) {
        const int g = idx / V, i = idx - g * V;
        v_pages[(place + (long)g * page_size) * V + i] = v[idx];
    }
}

// ---------------------------------------------------------------------------------------------------------------
// Rows of [q heads | k heads | v heads] (head widths D, D, V) of an attention that rotates part of its heads and mixes
// its values with another layer's:
//   the first rot elements of every q and k head turned by the token's angles (cos_sin [tokens][rot / 2][2]; pairing 0:
//   pairs (i, i + rot / 2), 1: neighbours; cos_sin == nullptr: none), q in place, k straight into its page;
//   v <- (1 - lambda) v + lambda v_first (v_first: row views of the same token's values in the other layer; nullptr:
//   v as it is), into its page.  The rows' own v stays as projected, for the layers that read it as v_first.
// One block a token; items of N elements (of both partners of a pair): N = 1, or 16 bytes where widths and rows allow.
template <typename T, int N> struct Items {      // N elements as 32-bit values
    static __device__ __forceinline__ void load(const T* p, float* o) { o[0] = to_f32(*p); }
    static __device__ __forceinline__ void store(T* p, const float* o) { *p = from_f32<T>(o[0]); }
};
template <> struct Items<float, 4> : Pack<float> {};
template <> struct Items<bf16, 8> : Pack<bf16> {};

template <typename T, int N>
__global__ void rotary_mix_store_kernel(T* __restrict__ qkv, long ld, const int* __restrict__ positions,
                                        const int* __restrict__ token_seq, const int* __restrict__ seq_slot,
                                        const float* __restrict__ cos_sin, int rot, int pairing,
                                        const T* __restrict__ v_first, long ld_first, float lambda,
                                        T* __restrict__ k_pages, T* __restrict__ v_pages,
                                        const int* __restrict__ block_table, int table_width, int page_size, int H, int G,
                                        int D, int V, int write_cache, int* __restrict__ status)
{
    fx_pdl_wait();
    const int t = blockIdx.x;
    const int pos = positions[t];
    T* row = qkv + (long)t * ld;
    long place = -1;      // (page, kv head 0, position in the page) as one index
    if (write_cache) {
        const int page = block_table[(long)seq_slot[token_seq[t]] * table_width + pos / page_size];
        if (page < 0) { if (threadIdx.x == 0 && status) atomicExch(status, 2); }
        else place = (long)page * G * page_size + (pos % page_size);
    }
    const int half = cos_sin ? rot >> 1 : 0;
    const float* cs = cos_sin + (long)t * half * 2;
    const int per_head = half / N;                  // rotated items of a head
    const int rest = (D - 2 * half) / N;            // and those that pass unchanged (k heads only: they are copied)
    const int n_q = H * per_head, n_k = G * (per_head + rest), n_v = G * (V / N);
    for (int idx = threadIdx.x; idx < n_q + n_k + n_v; idx += blockDim.x) {
        if (idx < n_q + n_k) {
            const bool is_q = idx < n_q;
            const int j = is_q ? idx : idx - n_q, per = is_q ? per_head : per_head + rest;
            const int h = j / per, c = j - h * per;
            T* x = row + (long)(is_q ? h : H + h) * D;
            T* dst = is_q ? x : place >= 0 ? k_pages + (place + (long)h * page_size) * D : nullptr;
            if (!dst) continue;
            if (c >= per_head) {      // beyond the rotated part
                const int i = 2 * half + (c - per_head) * N;
                float a[N];
                Items<T, N>::load(x + i, a);
                Items<T, N>::store(dst + i, a);
            } else if (pairing == 0) {
                const int i = c * N;
                float a[N], b[N], ra[N], rb[N];
                Items<T, N>::load(x + i, a);
                Items<T, N>::load(x + i + half, b);
#pragma unroll
                for (int e = 0; e < N; ++e) {
                    const float2 f = *reinterpret_cast<const float2*>(cs + (i + e) * 2);
                    ra[e] = a[e] * f.x - b[e] * f.y;
                    rb[e] = b[e] * f.x + a[e] * f.y;
                }
                Items<T, N>::store(dst + i, ra);
                Items<T, N>::store(dst + i + half, rb);
            } else {                  // (neighbours: N is 1)
                const float2 f = *reinterpret_cast<const float2*>(cs + c * 2);
                const float a = to_f32(x[2 * c]), b = to_f32(x[2 * c + 1]);
                dst[2 * c] = from_f32<T>(a * f.x - b * f.y);
                dst[2 * c + 1] = from_f32<T>(b * f.x + a * f.y);
            }
        } else if (place >= 0) {
            const int j = idx - n_q - n_k, per = V / N;
            const int g = j / per, i = (j - g * per) * N;
            float a[N];
            Items<T, N>::load(row + (long)(H + G) * D + (long)g * V + i, a);
            if (v_first) {
                float b[N];
                Items<T, N>::load(v_first + (long)t * ld_first + (long)g * V + i, b);
#pragma unroll
                for (int e = 0; e < N; ++e) a[e] = (1.0f - lambda) * a[e] + lambda * b[e];
            }
            Items<T, N>::store(v_pages + (place + (long)g * page_size) * V + i, a);
        }
    }
}

// ---------------------------------------------------------------------------------------------------------------
// Rows of [q heads | k heads | v heads] (head widths D, D, V) of an attention that norms its queries and keys behind the
// rotation and caches its values turned by their position:
//   q, k: the first rot elements of a head turned by the token's angles (cos_sin [tokens][rot / 2][2]; pairing as above;
//   nullptr: none), then, eps >= 0, x / sqrt(mean(x^2) + eps) over the head; q in place, k into its page;
//   v: pairs (2m, 2m + 1) of the whole head turned by v_cos_sin [tokens][V / 2][2] (nullptr: as it is), into its page.
// The rows' own k and v stay as projected.  A warp a head (the head's row as 32-bit values in shared memory), gridDim.y
// blocks a token; items of N elements.
template <> struct Items<bf16, 4> {
    static __device__ __forceinline__ void load(const bf16* p, float* o) {
        const uint2 v = *reinterpret_cast<const uint2*>(p);
        o[0] = __uint_as_float(v.x << 16); o[1] = __uint_as_float(v.x & 0xffff0000u);
        o[2] = __uint_as_float(v.y << 16); o[3] = __uint_as_float(v.y & 0xffff0000u);
    }
    static __device__ __forceinline__ void store(bf16* p, const float* o) {
        __nv_bfloat162 a = __floats2bfloat162_rn(o[0], o[1]), b = __floats2bfloat162_rn(o[2], o[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
    }
};

constexpr int RN_WARPS = 8;

template <typename T, int N>
__global__ void __launch_bounds__(RN_WARPS * 32) rotary_norm_store_kernel(
    T* __restrict__ qkv, long ld, const int* __restrict__ positions, const int* __restrict__ token_seq,
    const int* __restrict__ seq_slot, const float* __restrict__ cos_sin, int rot, int pairing, float eps,
    const float* __restrict__ v_cos_sin, T* __restrict__ k_pages, T* __restrict__ v_pages,
    const int* __restrict__ block_table, int table_width, int page_size, int H, int G, int D, int V, int write_cache,
    int* __restrict__ status)
{
    extern __shared__ __align__(16) float rn_s[];
    fx_pdl_wait();
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int pos = positions[t];
    T* row = qkv + (long)t * ld;
    long place = -1;      // (page, kv head 0, position in the page) as one index
    if (write_cache) {
        const int page = block_table[(long)seq_slot[token_seq[t]] * table_width + pos / page_size];
        if (page < 0) { if (threadIdx.x == 0 && status) atomicExch(status, 2); }
        else place = (long)page * G * page_size + (pos % page_size);
    }
    float* x_s = rn_s + warp * (((D > V ? D : V) + 3) & ~3);
    const int half = rot >> 1;
    const float* cs = cos_sin ? cos_sin + (long)t * half * 2 : nullptr;
    const float* vcs = v_cos_sin ? v_cos_sin + (long)t * V : nullptr;
    const int units = H + 2 * G;
    for (int u = blockIdx.y * RN_WARPS + warp; u < units; u += gridDim.y * RN_WARPS) {
        const bool is_q = u < H, is_v = u >= H + G;
        if (!is_q && place < 0) continue;
        const int width = is_v ? V : D;
        T* x = row + (is_v ? (long)(H + G) * D + (long)(u - H - G) * V : (long)u * D);
        T* dst = is_q ? x : is_v ? v_pages + (place + (long)(u - H - G) * page_size) * V
                                 : k_pages + (place + (long)(u - H) * page_size) * D;
        float ss = 0.f;
        for (int i = lane * N; i < width; i += 32 * N) {
            float a[N];
            Items<T, N>::load(x + i, a);
#pragma unroll
            for (int e = 0; e < N; ++e) { x_s[i + e] = a[e]; ss = fmaf(a[e], a[e], ss); }
        }
        __syncwarp();
        // (a rotation leaves the sum of squares as it is)
        const float r = is_v || eps < 0.f ? 1.f : 1.0f / sqrtf(warp_sum(ss) / (float)D + eps);
        for (int i = lane * N; i < width; i += 32 * N) {
            float a[N];
#pragma unroll
            for (int e = 0; e < N; ++e) {
                const int j = i + e;
                const float own = x_s[j];
                float y = own;
                if (is_v) {
                    if (vcs) {
                        const float2 f = *reinterpret_cast<const float2*>(vcs + (j & ~1));
                        const float other = x_s[j ^ 1];
                        y = j & 1 ? own * f.x + other * f.y : own * f.x - other * f.y;
                    }
                } else if (cs && j < rot) {
                    const bool second = pairing ? j & 1 : j >= half;
                    const int p = pairing ? j >> 1 : (second ? j - half : j);
                    const float2 f = *reinterpret_cast<const float2*>(cs + p * 2);
                    const float other = x_s[pairing ? j ^ 1 : (second ? j - half : j + half)];
                    y = second ? own * f.x + other * f.y : own * f.x - other * f.y;
                }
                a[e] = y * r;
            }
            Items<T, N>::store(dst + i, a);
        }
        __syncwarp();
    }
}

// The same for heads of up to 128 elements rotated on pairs (i, i + rot / 2) whose halves are whole pieces of four: a lane
// holds its piece of the head and, where that is rotated, the partner piece, in registers; nothing passes through shared
// memory.  (A query head is written over itself: every lane has its pieces before the sum over the warp.)
template <typename T>
__global__ void __launch_bounds__(RN_WARPS * 32) rotary_norm_store_128_kernel(
    T* __restrict__ qkv, long ld, const int* __restrict__ positions, const int* __restrict__ token_seq,
    const int* __restrict__ seq_slot, const float* __restrict__ cos_sin, int rot, float eps,
    const float* __restrict__ v_cos_sin, T* __restrict__ k_pages, T* __restrict__ v_pages,
    const int* __restrict__ block_table, int table_width, int page_size, int H, int G, int D, int V, int write_cache,
    int* __restrict__ status)
{
    fx_pdl_wait();
    const int t = blockIdx.x, i = (threadIdx.x & 31) * 4, warp = threadIdx.x >> 5;
    const int u = blockIdx.y * RN_WARPS + warp;
    if (u >= H + 2 * G) return;      // (whole warps; no barrier below)
    const bool is_q = u < H, is_v = u >= H + G;
    T* x = qkv + (long)t * ld + (is_v ? (long)(H + G) * D + (long)(u - H - G) * V : (long)u * D);
    T* dst = x;
    if (!is_q) {
        if (!write_cache) return;
        const int pos = positions[t], p = pos / page_size;
        const int page = block_table[(long)seq_slot[token_seq[t]] * table_width + p];
        if (page < 0) { if ((threadIdx.x & 31) == 0 && status) atomicExch(status, 2); return; }
        const int g = is_v ? u - H - G : u - H;
        dst = (is_v ? v_pages : k_pages) + (((long)page * G + g) * page_size + (pos - p * page_size)) * (is_v ? V : D);
    }
    const int width = is_v ? V : D, half = cos_sin ? rot >> 1 : 0;
    const bool in = i < width;
    float a[4] = {0.f, 0.f, 0.f, 0.f};
    if (in) Items<T, 4>::load(x + i, a);
    if (is_v) {
        if (!in) return;
        if (v_cos_sin) {
            const float4 f = *reinterpret_cast<const float4*>(v_cos_sin + (long)t * V + i);      // (two pairs)
            const float b0 = a[0], b2 = a[2];
            a[0] = b0 * f.x - a[1] * f.y; a[1] = a[1] * f.x + b0 * f.y;
            a[2] = b2 * f.z - a[3] * f.w; a[3] = a[3] * f.z + b2 * f.w;
        }
        Items<T, 4>::store(dst + i, a);
        return;
    }
    float b[4] = {0.f, 0.f, 0.f, 0.f};
    const bool turned = i < 2 * half, second = i >= half;
    if (turned) Items<T, 4>::load(x + (second ? i - half : i + half), b);
    if (eps >= 0.f) {      // (a rotation leaves the sum of squares as it is)
        const float ss = warp_sum(fmaf(a[0], a[0], fmaf(a[1], a[1], fmaf(a[2], a[2], a[3] * a[3]))));
        const float r = 1.0f / sqrtf(ss / (float)D + eps);
#pragma unroll
        for (int e = 0; e < 4; ++e) { a[e] *= r; b[e] *= r; }
    }
    __syncwarp();
    if (!in) return;
    if (turned) {
        const float* cs = cos_sin + ((long)t * half + (second ? i - half : i)) * 2;
        const float4 f0 = *reinterpret_cast<const float4*>(cs), f1 = *reinterpret_cast<const float4*>(cs + 4);
        const float sg = second ? 1.f : -1.f;
        a[0] = a[0] * f0.x + sg * b[0] * f0.y; a[1] = a[1] * f0.z + sg * b[1] * f0.w;
        a[2] = a[2] * f1.x + sg * b[2] * f1.y; a[3] = a[3] * f1.z + sg * b[3] * f1.w;
    }
    Items<T, 4>::store(dst + i, a);
}

// ---------------------------------------------------------------------------------------------------------------
// The latent form.  Per token: `dkv` = [C latent | R rotated key part] as projected, `q` = H heads of [D | R].
//   c <- dkv[:C] / sqrt(mean(dkv[:C]^2) + eps) * wc            -> pages[position][0:C]
//   k_rot <- pairs (2i, 2i+1) of the first rot_dims of dkv[C:] turned by the position's angles, the rest as it is
//                                                               -> pages[position][C:C+R]
//   q's D part of every head                                    -> q_plain[head][token][0:D]      (head by head)
//   q's R part of every head, turned the same way               -> q_full[head][token][C:C+R]
// q_full's first C columns are filled afterwards by the product of q_plain with the keys' read-out matrix, so that a
// score is one dot product of C + R elements against a cached row.  cos_sin: [tokens][rot_dims / 2][2].
// q_plain == nullptr: the queries stay token rows and only their rotated parts are turned, in place (the form in
// which keys and values are read out of the latent before the attention).
// One block a token.
template <typename T>
__global__ void latent_prep_kernel(T* __restrict__ q, long ldq, const T* __restrict__ dkv, long ld_dkv,
                                   const int* __restrict__ positions, const int* __restrict__ token_seq,
                                   const int* __restrict__ seq_slot, const void* __restrict__ wc, int w_dtype, float eps,
                                   const float* __restrict__ cos_sin, int rot_dims, T* __restrict__ q_plain,
                                   T* __restrict__ q_full, T* __restrict__ pages, const int* __restrict__ block_table,
                                   int table_width, int page_size, int n_tokens, int H, int D, int R, int C,
                                   int write_cache, int* __restrict__ status, int pairing)
{
    // pairing 1: neighbours (2i, 2i + 1); 0: halves (i, i + rot_dims / 2).  Thread i < half turns pair i; the
    // threads beyond copy element rot_dims + (i - half).
    __shared__ float scratch[33];
    fx_pdl_wait();
    const int t = blockIdx.x;
    const int pos = positions[t];
    const int half = rot_dims >> 1;
    const float* cs = cos_sin + (long)t * half * 2;
    const int W = C + R;
    const T* d = dkv + (long)t * ld_dkv;
    T* dst = nullptr;
    if (write_cache) {
        const int page = block_table[(long)seq_slot[token_seq[t]] * table_width + pos / page_size];
        if (page < 0) { if (threadIdx.x == 0 && status) atomicExch(status, 2); }
        else dst = pages + ((long)page * page_size + (pos % page_size)) * W;
    }
    // queries: the plain part head by head, the rotated part into its place behind the latent columns
    T* qr = q + (long)t * ldq;
    if (q_plain)
        for (int idx = threadIdx.x; idx < H * D; idx += blockDim.x) {
            const int h = idx / D, i = idx - h * D;
            q_plain[((long)h * n_tokens + t) * D + i] = qr[(long)h * (D + R) + i];
        }
    for (int idx = threadIdx.x; idx < H * (R - half); idx += blockDim.x) {
        const int h = idx / (R - half), i = idx - h * (R - half);
        T* x = qr + (long)h * (D + R) + D;
        T* o = q_plain ? q_full + ((long)h * n_tokens + t) * W + C : x;   // no head-by-head copy: turned where it lies
        if (i < half) {
            const int ia = pairing ? 2 * i : i, ib = pairing ? 2 * i + 1 : i + half;
            const float a = to_f32(x[ia]), b = to_f32(x[ib]), c = cs[2 * i], s = cs[2 * i + 1];
            o[ia] = from_f32<T>(a * c - b * s);
            o[ib] = from_f32<T>(b * c + a * s);
        } else {
            o[half + i] = x[half + i];      // beyond the rotated pairs: element rot_dims + (i - half)
        }
    }
    if (!dst) return;    // (uniform across the block)
    float ss = 0.f;
    for (int i = threadIdx.x; i < C; i += blockDim.x) { const float v = to_f32(d[i]); ss = fmaf(v, v, ss); }
    ss = block_sum(ss, scratch);
    const float r = sqrtf(ss / (float)C + eps);
    for (int i = threadIdx.x; i < C; i += blockDim.x)
        dst[i] = from_f32<T>(to_f32(d[i]) / r * load_any(wc, w_dtype, i));
    for (int i = threadIdx.x; i < R - half; i += blockDim.x) {
        const T* x = d + C;
        if (i < half) {
            const int ia = pairing ? 2 * i : i, ib = pairing ? 2 * i + 1 : i + half;
            const float a = to_f32(x[ia]), b = to_f32(x[ib]), c = cs[2 * i], s = cs[2 * i + 1];
            dst[C + ia] = from_f32<T>(a * c - b * s);
            dst[C + ib] = from_f32<T>(b * c + a * s);
        } else {
            dst[C + half + i] = x[half + i];
        }
    }
}

// out[t, :] = x[t, :] / sqrt(mean(x[t, :]^2) + eps) * w over rows with strides; one block a row.
template <typename TI, typename TO>
__global__ void rmsnorm_rows_kernel(const TI* __restrict__ x, long ldx, const void* __restrict__ w, int w_dtype, float eps,
                                    TO* __restrict__ out, long ldo, int n)
{
    __shared__ float scratch[33];
    fx_pdl_wait();
    const TI* xr = x + (long)blockIdx.x * ldx;
    float ss = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) { const float v = to_f32(xr[i]); ss = fmaf(v, v, ss); }
    ss = block_sum(ss, scratch);
    const float r = sqrtf(ss / (float)n + eps);
    TO* o = out + (long)blockIdx.x * ldo;
    for (int i = threadIdx.x; i < n; i += blockDim.x) o[i] = from_f32<TO>(to_f32(xr[i]) / r * load_any(w, w_dtype, i));
}

// out[t][h * V + v] = in[t * in_ldt + h * in_ldh + v] * (gate ? sigmoid(gate[t][h * V + v]) : 1): rows laid out head
// by head ([h][t][v]: in_ldh = tokens * V, in_ldt = V) back into token rows, with the output gate of the mixer applied
// (gate_per_head: one gate a head, gate[t][h], instead of one an element)
// on the way; or token rows gated where they lie (in == out, in_ldt = ldo, in_ldh = V).
template <typename T>
__global__ void heads_to_tokens_kernel(const T* in, long in_ldt, long in_ldh, const T* __restrict__ gate, long ldg, T* out,
                                       long ldo, int n_tokens, int H, int V, int gate_per_head)
{
    fx_pdl_wait();
    const long total = (long)n_tokens * H * V;
    for (long idx = blockIdx.x * (long)blockDim.x + threadIdx.x; idx < total; idx += (long)gridDim.x * blockDim.x) {
        const int t = (int)(idx / (H * V));
        const int c = (int)(idx - (long)t * H * V);
        const int h = c / V, v = c - h * V;
        float x = to_f32(in[(long)t * in_ldt + (long)h * in_ldh + v]);
        if (gate) x *= 1.0f / (1.0f + expf(-to_f32(gate[(long)t * ldg + (gate_per_head ? h : c)])));
        out[(long)t * ldo + c] = from_f32<T>(x);
    }
}

int threads_for_width(int n) {
    int t = 32;
    while (t < n && t < 256) t <<= 1;
    return t;
}

}  // namespace

extern "C" int fx_qk_norm_store(void* qkv, int dtype, long ld, const int* positions, const int* token_seq,
                                const int* seq_slot, const void* wq, const void* wk, int w_dtype, float eps,
                                float temp_coef, int temp_every, void* k_pages, void* v_pages, const int* block_table,
                                int table_width, int page_size, int n_tokens, int n_heads, int n_kv_heads, int key_dim,
                                int value_dim, int write_cache, int* status, float v_eps, void* stream)
{
    if (n_tokens <= 0) return FX_OK;
    if (key_dim <= 0 || value_dim <= 0 || page_size <= 0 || n_heads <= 0 || n_kv_heads <= 0) return FX_ERR_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    const int nt = 32 * (n_heads + n_kv_heads > 8 ? 8 : n_heads + n_kv_heads);
#define FX_GO(T)                                                                                                      \
    fx_launch_pdl(qk_norm_store_kernel<T>, n_tokens, nt, 0, s, (T*)qkv, ld, positions, token_seq, seq_slot, wq, wk,  \
                  w_dtype, eps, temp_coef, temp_every, (T*)k_pages, (T*)v_pages, block_table, table_width, page_size, \
                  n_heads, n_kv_heads, key_dim, value_dim, write_cache, status, v_eps)
    if (dtype == FX_F32) FX_GO(float);
    else if (dtype == FX_BF16) FX_GO(bf16);
    else return FX_ERR_DTYPE;
#undef FX_GO
    return fx_launch_status();
}

extern "C" int fx_rotary_mix_store(void* qkv, int dtype, long ld, const int* positions, const int* token_seq,
                                   const int* seq_slot, const float* cos_sin, int rot, int pairing, const void* v_first,
                                   long ld_first, float lambda, void* k_pages, void* v_pages, const int* block_table,
                                   int table_width, int page_size, int n_tokens, int n_heads, int n_kv_heads, int key_dim,
                                   int value_dim, int write_cache, int* status, void* stream)
{
    if (n_tokens <= 0) return FX_OK;
    if (key_dim <= 0 || value_dim <= 0 || page_size <= 0 || n_heads <= 0 || n_kv_heads <= 0 || pairing < 0 || pairing > 1)
        return FX_ERR_SIZE;
    if (!cos_sin) rot = 0;
    if (rot < 0 || rot % 2 || rot > key_dim) return FX_ERR_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    const int vw = dtype == FX_F32 ? 4 : 8;
    const int es = dtype == FX_F32 ? 4 : 2;
    const bool vec = pairing == 0 && (rot / 2) % vw == 0 && key_dim % vw == 0 && value_dim % vw == 0 && (ld * es) % 16 == 0 &&
                     (ld_first * es) % 16 == 0 && (uintptr_t)qkv % 16 == 0 && (uintptr_t)v_first % 16 == 0 &&
                     (uintptr_t)k_pages % 16 == 0 && (uintptr_t)v_pages % 16 == 0;
    const int n = vec ? vw : 1;
    const int items = (n_heads * (rot / 2) + n_kv_heads * (key_dim - rot / 2 + value_dim)) / n;
    const int nt = threads_for_width(items);
#define FX_GO(T, N)                                                                                                   \
    fx_launch_pdl(rotary_mix_store_kernel<T, N>, n_tokens, nt, 0, s, (T*)qkv, ld, positions, token_seq, seq_slot,    \
                  cos_sin, rot, pairing, (const T*)v_first, ld_first, lambda, (T*)k_pages, (T*)v_pages, block_table, \
                  table_width, page_size, n_heads, n_kv_heads, key_dim, value_dim, write_cache, status)
    if (dtype == FX_F32) { if (vec) FX_GO(float, 4); else FX_GO(float, 1); }
    else if (dtype == FX_BF16) { if (vec) FX_GO(bf16, 8); else FX_GO(bf16, 1); }
    else return FX_ERR_DTYPE;
#undef FX_GO
    return fx_launch_status();
}

// eps < 0: queries and keys are not normed.  Refuses (FX_ERR_SIZE) heads wider than the shared memory holds.
extern "C" int fx_rotary_norm_store(void* qkv, int dtype, long ld, const int* positions, const int* token_seq,
                                    const int* seq_slot, const float* cos_sin, int rot, int pairing, float eps,
                                    const float* v_cos_sin, void* k_pages, void* v_pages, const int* block_table,
                                    int table_width, int page_size, int n_tokens, int n_heads, int n_kv_heads,
                                    int key_dim, int value_dim, int write_cache, int* status, void* stream)
{
    if (n_tokens <= 0) return FX_OK;
    if (key_dim <= 0 || value_dim <= 0 || page_size <= 0 || n_heads <= 0 || n_kv_heads <= 0 || pairing < 0 || pairing > 1)
        return FX_ERR_SIZE;
    if (!cos_sin) rot = 0;
    if (rot < 0 || rot % 2 || rot > key_dim || (v_cos_sin && value_dim % 2)) return FX_ERR_SIZE;
    if ((uintptr_t)cos_sin % 8 || (uintptr_t)v_cos_sin % 8) return FX_ERR_ALIGN;
    const int widest = ((key_dim > value_dim ? key_dim : value_dim) + 3) & ~3;
    const size_t smem = (size_t)RN_WARPS * widest * 4;
    if (smem > 48 * 1024) return FX_ERR_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    const int item = dtype == FX_F32 ? 16 : 8;     // bytes of four elements
    const bool vec = key_dim % 4 == 0 && value_dim % 4 == 0 && ld % 4 == 0 && (uintptr_t)qkv % item == 0 &&
                     (uintptr_t)k_pages % item == 0 && (uintptr_t)v_pages % item == 0;
    const int units = n_heads + 2 * n_kv_heads;
    dim3 grid(n_tokens, (unsigned)fx_cdiv(units, RN_WARPS));      // (a warp a head)
#define FX_GO(T, N)                                                                                                   \
    fx_launch_pdl(rotary_norm_store_kernel<T, N>, grid, RN_WARPS * 32, smem, s, (T*)qkv, ld, positions, token_seq,   \
                  seq_slot, cos_sin, rot, pairing, eps, v_cos_sin, (T*)k_pages, (T*)v_pages, block_table, table_width, \
                  page_size, n_heads, n_kv_heads, key_dim, value_dim, write_cache, status)
    if (vec && pairing == 0 && rot % 8 == 0 && key_dim <= 128 && value_dim <= 128 && (uintptr_t)cos_sin % 16 == 0 &&
        (uintptr_t)v_cos_sin % 16 == 0) {
#define FX_GO128(T)                                                                                                   \
    fx_launch_pdl(rotary_norm_store_128_kernel<T>, grid, RN_WARPS * 32, 0, s, (T*)qkv, ld, positions, token_seq,     \
                  seq_slot, cos_sin, rot, eps, v_cos_sin, (T*)k_pages, (T*)v_pages, block_table, table_width, page_size, \
                  n_heads, n_kv_heads, key_dim, value_dim, write_cache, status)
        if (dtype == FX_F32) FX_GO128(float);
        else if (dtype == FX_BF16) FX_GO128(bf16);
        else return FX_ERR_DTYPE;
#undef FX_GO128
        return fx_launch_status();
    }
    if (dtype == FX_F32) { if (vec) FX_GO(float, 4); else FX_GO(float, 1); }
    else if (dtype == FX_BF16) { if (vec) FX_GO(bf16, 4); else FX_GO(bf16, 1); }
    else return FX_ERR_DTYPE;
#undef FX_GO
    return fx_launch_status();
}

extern "C" int fx_latent_prep(void* q, long ldq, const void* dkv, long ld_dkv, int dtype, const int* positions,
                              const int* token_seq, const int* seq_slot, const void* wc, int w_dtype, float eps,
                              const float* cos_sin, int rot_dims, void* q_plain, void* q_full, void* pages,
                              const int* block_table, int table_width, int page_size, int n_tokens, int n_heads,
                              int plain_dim, int rot_dim, int rank, int write_cache, int* status, int pairing,
                              void* stream)
{
    if (n_tokens <= 0) return FX_OK;
    if (pairing < 0 || pairing > 1) return FX_ERR_SIZE;
    if (rot_dims % 2 || rot_dims > rot_dim || rot_dims < 0 || plain_dim <= 0 || rank <= 0 || page_size <= 0)
        return FX_ERR_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    const int nt = threads_for_width(n_heads * plain_dim > rank ? n_heads * plain_dim : rank);
#define FX_GO(T)                                                                                                      \
    fx_launch_pdl(latent_prep_kernel<T>, n_tokens, nt, 0, s, (T*)q, ldq, (const T*)dkv, ld_dkv, positions,      \
                  token_seq, seq_slot, wc, w_dtype, eps, cos_sin, rot_dims, (T*)q_plain, (T*)q_full, (T*)pages,       \
                  block_table, table_width, page_size, n_tokens, n_heads, plain_dim, rot_dim, rank, write_cache, status, pairing)
    if (dtype == FX_F32) FX_GO(float);
    else if (dtype == FX_BF16) FX_GO(bf16);
    else return FX_ERR_DTYPE;
#undef FX_GO
    return fx_launch_status();
}

extern "C" int fx_rmsnorm_rows(const void* x, int x_dtype, long ldx, const void* w, int w_dtype, float eps, void* out,
                               int out_dtype, long ldo, int n_rows, int n, void* stream)
{
    if (n_rows <= 0 || n <= 0) return FX_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const int nt = threads_for_width(n);
#define FX_GO(TI, TO)                                                                                                 \
    fx_launch_pdl(rmsnorm_rows_kernel<TI, TO>, n_rows, nt, 0, s, (const TI*)x, ldx, w, w_dtype, eps, (TO*)out, ldo, n)
    if (x_dtype == FX_F32 && out_dtype == FX_F32) FX_GO(float, float);
    else if (x_dtype == FX_F32 && out_dtype == FX_BF16) FX_GO(float, bf16);
    else if (x_dtype == FX_BF16 && out_dtype == FX_BF16) FX_GO(bf16, bf16);
    else if (x_dtype == FX_BF16 && out_dtype == FX_F32) FX_GO(bf16, float);
    else return FX_ERR_DTYPE;
#undef FX_GO
    return fx_launch_status();
}

extern "C" int fx_heads_to_tokens(const void* in, long in_ldt, long in_ldh, const void* gate, long ldg, void* out, long ldo,
                                  int dtype, int n_tokens, int n_heads, int width, int gate_per_head, void* stream)
{
    if (n_tokens <= 0 || n_heads <= 0 || width <= 0) return FX_OK;
    cudaStream_t s = (cudaStream_t)stream;
    long blocks = fx_cdiv((long)n_tokens * n_heads * width, 256);
    if (blocks > fx_sm_count() * 16L) blocks = fx_sm_count() * 16L;
    if (dtype == FX_F32)
        fx_launch_pdl(heads_to_tokens_kernel<float>, (unsigned)blocks, 256, 0, s, (const float*)in, in_ldt, in_ldh, (const float*)gate, ldg,
                      (float*)out, ldo, n_tokens, n_heads, width, gate_per_head);
    else if (dtype == FX_BF16)
        fx_launch_pdl(heads_to_tokens_kernel<bf16>, (unsigned)blocks, 256, 0, s, (const bf16*)in, in_ldt, in_ldh, (const bf16*)gate, ldg,
                      (bf16*)out, ldo, n_tokens, n_heads, width, gate_per_head);
    else return FX_ERR_DTYPE;
    return fx_launch_status();
}
