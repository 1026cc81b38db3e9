// Linear attention whose state decays channel by channel: per head a matrix S [dim (keys), vdim (values)],
//
//   S <- diag(alpha) S + k v^T,    o = q_scale S^T q,    alpha = sigmoid(w2 . low + bias)^(1/tau)
//
// over the tokens of a request in order.  Everything here is 32-bit CUDA-core arithmetic: state, decays, products.
//
// fx_channel_decay_prep makes alpha of every (token, key channel) from the low-rank rows.
//
// fx_channel_decay_scan: nothing couples two columns (values) of S, nor two rows but for the read-out, so the loop over
// the tokens has no exchange between threads at all.  A block of 256 threads owns CD_COLS columns of one head of one
// request: a lane one column, sixteen groups of rows (a half-warp each) RPL rows of it in registers.  q, k and alpha of a
// group's rows are the same for all its lanes, so shared memory is read as broadcasts, sixteen bytes at a time.  The
// tokens' rows travel into shared memory CD_CH tokens at a time by cp.async, the next chunk while this one is worked on;
// the groups' shares of the read-outs are added up once a chunk.  The order of additions does not depend on how a
// request was cut into steps.  State [slots, H, D, V]: a row's columns lie together.
//
// fx_fixed_decay_scan: the same loop for one fixed decay a head, S <- d S + k v^T (the recurrence of fx_state_scan without
// its delta rule, over a state laid out as there, column by column), for long prompts.
#include "common.cuh"
#include "api.h"

namespace {

// first row r with token_seq[r] >= b
__device__ __forceinline__ int first_row_of(const int* __restrict__ token_seq, int n_tokens, int b)
{
    int lo = 0, hi = n_tokens;
    while (lo < hi) {
        const int mid = (lo + hi) >> 1;
        if (token_seq[mid] < b) lo = mid + 1; else hi = mid;
    }
    return lo;
}

// sigmoid(z)^p = e^-a with a = p log(1 + e^-z): close to 1 the exponent keeps its relative precision.  The decay is raised
// to the power of the distance a memory travels, so that a bias in its last place grows a thousandfold over a thousand
// tokens: where a is small, e^-a is 1 plus e^-a - 1 from its Taylor series, rounded once.
__device__ __forceinline__ float sigmoid_power(float z, float p)
{
    const float a = -p * fx_softplus(-z);
    // a > -1/8: e^a - 1 = a (1 + a/2 (1 + a/3 (1 + a/4 (1 + a/5)))), the next term below 5e-8 of the sum
    float q = fmaf(a, 1.0f / 120.0f, 1.0f / 24.0f);
    q = fmaf(q, a, 1.0f / 6.0f);
    q = fmaf(q, a, 0.5f);
    q = fmaf(q, a, 1.0f);
    return a > -0.125f ? fmaf(q, a, 1.0f) : expf(a);
}

constexpr int CP_THREADS = 128;
constexpr int CP_TOKENS = 8;
constexpr int CP_RC = 128;      // low-rank channels a pass

// One block: CP_TOKENS tokens, CP_THREADS channels, a channel a thread.
__global__ void __launch_bounds__(CP_THREADS) channel_decay_prep_kernel(
    const float* __restrict__ low, long ldl, const void* __restrict__ w2, int w2_dtype, const void* __restrict__ bias,
    int b_dtype, float inv_tau, float* __restrict__ alpha, int n_tokens, int C, int rank)
{
    __shared__ float low_s[CP_RC][CP_TOKENS];
    fx_pdl_wait();
    const int t0 = blockIdx.x * CP_TOKENS, c = blockIdx.y * CP_THREADS + threadIdx.x;
    const int nt = min(CP_TOKENS, n_tokens - t0);
    float z[CP_TOKENS];
#pragma unroll
    for (int i = 0; i < CP_TOKENS; ++i) z[i] = 0.f;
    for (int r0 = 0; r0 < rank; r0 += CP_RC) {
        const int nr = min(CP_RC, rank - r0);
        __syncthreads();
        for (int idx = threadIdx.x; idx < nr * CP_TOKENS; idx += CP_THREADS) {
            const int tt = idx / nr, r = idx - tt * nr;
            low_s[r][tt] = tt < nt ? low[(long)(t0 + tt) * ldl + r0 + r] : 0.f;
        }
        __syncthreads();
        if (c < C)
            for (int r = 0; r < nr; ++r) {
                const float w = load_any(w2, w2_dtype, (long)c * rank + r0 + r);
#pragma unroll
                for (int i = 0; i < CP_TOKENS; ++i) z[i] = fmaf(w, low_s[r][i], z[i]);
            }
    }
    if (c >= C) return;
    const float b = load_any(bias, b_dtype, c);
#pragma unroll
    for (int i = 0; i < CP_TOKENS; ++i)
        if (i < nt) alpha[(long)(t0 + i) * C + c] = sigmoid_power(z[i] + b, inv_tau);
}

constexpr int CD_THREADS = 256;
constexpr int CD_COLS = 16;                            // columns a block
constexpr int CD_GROUPS = CD_THREADS / CD_COLS;        // groups of rows
constexpr int CD_CH = 16;                              // tokens a chunk
constexpr int CD_MAX_D = 256;

__device__ __forceinline__ void cp_async4(uint32_t dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

struct CdArgs {
    const float* src[3];   // rows of q, k, alpha: the head's D elements of token t at src[i] + t * ld[i] + h * D
    long ld[3];
    const float* v; long ldv;
    float q_scale;
    const float* decay;    // one fixed decay a head (no alpha rows then)
    float* state;          // [slots, H][D, V], row i, column j of a head at i * row_stride + j * col_stride
    long row_stride, col_stride;
    float* out; long ldo;  // [T, H * V]
    const int *token_seq, *seq_slot;
    int n_tokens, H, D, V;
    int vec;               // q, k, alpha rows may be copied 16 bytes at a time
};

// Shared memory: two buffers of [3][CD_CH][DP] rows (FIXED: [2]) and [CD_CH][CD_COLS] values, then [CD_CH][CD_GROUPS][CD_COLS]
// read-out shares; DP = RPL * CD_GROUPS.
template <int RPL, bool FIXED>
__global__ void __launch_bounds__(CD_THREADS) channel_decay_scan_kernel(const CdArgs a)
{
    constexpr int DP = RPL * CD_GROUPS, ROWS = FIXED ? 2 : 3;
    constexpr int BUF = CD_CH * (ROWS * DP + CD_COLS);
    extern __shared__ __align__(16) float sm[];
    fx_pdl_wait_only();
    const int b = blockIdx.x, h = blockIdx.y, D = a.D;
    const int col = threadIdx.x % CD_COLS, grp = threadIdx.x / CD_COLS;
    const int col0 = blockIdx.z * CD_COLS, nc = min(CD_COLS, a.V - col0);
    const int r0 = first_row_of(a.token_seq, a.n_tokens, b), r1 = first_row_of(a.token_seq, a.n_tokens, b + 1);
    if (r1 <= r0) return;
    float* rd_s = sm + 2 * BUF;
    const uint32_t sm_u = (uint32_t)__cvta_generic_to_shared(sm);
    const bool live = col < nc;
    float* sp = a.state + ((long)a.seq_slot[b] * a.H + h) * D * a.V + (long)(col0 + (live ? col : 0)) * a.col_stride;
    const float fixed = FIXED ? a.decay[h] : 0.f;

    float S[RPL];
#pragma unroll
    for (int i = 0; i < RPL; ++i) {
        const int row = grp * RPL + i;
        S[i] = (live && row < D) ? sp[row * a.row_stride] : 0.f;
    }
    // what lies beyond the head's D rows and the live columns stays zero in both buffers
    if (D < DP || nc < CD_COLS) {
        for (int idx = threadIdx.x; idx < 2 * BUF; idx += CD_THREADS) sm[idx] = 0.f;
        __syncthreads();
    }

    // Staging.  Thread t copies piece t, t + 256, ... of a chunk; a piece's (token, place in the row) moves on by the
    // same step every time, so the quotient and the remainder are taken once and carried from piece to piece.
    const int pw = a.vec ? D >> 2 : D;                   // pieces a row: 16 bytes each, or one element
    const int p_tt0 = threadIdx.x / pw, p_i0 = threadIdx.x - p_tt0 * pw;
    const int p_dq = CD_THREADS / pw, p_dr = CD_THREADS - p_dq * pw;
    const float* srcp[ROWS];
#pragma unroll
    for (int arr = 0; arr < ROWS; ++arr) srcp[arr] = a.src[arr] + (long)h * D;
    const float* vp = a.v + (long)h * a.V + col0;
    auto issue = [&](int c0, int nt, int buf) {
        const uint32_t base = sm_u + (uint32_t)(buf * BUF) * 4u;
        for (int tt = p_tt0, i = p_i0; tt < nt;) {
            const int e = a.vec ? i * 4 : i;
#pragma unroll
            for (int arr = 0; arr < ROWS; ++arr) {
                const uint32_t dst = base + (uint32_t)((arr * CD_CH + tt) * DP + e) * 4u;
                const float* src = srcp[arr] + (long)(c0 + tt) * a.ld[arr] + e;
                if (a.vec) cp_async16(dst, src); else cp_async4(dst, src);
            }
            tt += p_dq; i += p_dr;
            if (i >= pw) { i -= pw; ++tt; }
        }
        const int tt = threadIdx.x / CD_COLS;            // (CD_CH * CD_COLS values: one a thread)
        if (tt < nt && live) cp_async4(base + (uint32_t)(ROWS * CD_CH * DP + threadIdx.x) * 4u, vp + (long)(c0 + tt) * a.ldv + col);
    };

    issue(r0, min(CD_CH, r1 - r0), 0);
    cp_commit();
    int buf = 0;
    for (int c0 = r0; c0 < r1; c0 += CD_CH, buf ^= 1) {
        const int nt = min(CD_CH, r1 - c0);
        if (c0 + CD_CH < r1) {
            issue(c0 + CD_CH, min(CD_CH, r1 - c0 - CD_CH), buf ^ 1);
            cp_commit();
            cp_wait<1>();
        } else {
            cp_wait<0>();
        }
        __syncthreads();
        const float* q_s = sm + buf * BUF + grp * RPL;
        const float* k_s = q_s + CD_CH * DP;
        const float* w_s = k_s + CD_CH * DP;
        const float* v_s = sm + buf * BUF + ROWS * CD_CH * DP + col;
        auto token = [&](int tt) {      // one token: the state moves on; this thread's share of the read-out
            const float vt = v_s[tt * CD_COLS];
            float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
#pragma unroll
            for (int i = 0; i < RPL; i += 4) {
                const float4 ww = FIXED ? make_float4(fixed, fixed, fixed, fixed) : *reinterpret_cast<const float4*>(w_s + tt * DP + i);
                const float4 kk = *reinterpret_cast<const float4*>(k_s + tt * DP + i);
                const float4 qq = *reinterpret_cast<const float4*>(q_s + tt * DP + i);
                S[i] = fmaf(ww.x, S[i], kk.x * vt); S[i + 1] = fmaf(ww.y, S[i + 1], kk.y * vt);
                S[i + 2] = fmaf(ww.z, S[i + 2], kk.z * vt); S[i + 3] = fmaf(ww.w, S[i + 3], kk.w * vt);
                d0 = fmaf(S[i], qq.x, d0); d1 = fmaf(S[i + 1], qq.y, d1);
                d2 = fmaf(S[i + 2], qq.z, d2); d3 = fmaf(S[i + 3], qq.w, d3);
            }
            return (d0 + d1) + (d2 + d3);
        };
        // Whole chunks by four tokens: the shares are stored after the four, so that the second's rows are asked for while
        // the first is worked on (a store to shared memory between them would hold the loads back).
        int tt = 0;
        for (; tt + 4 <= nt; tt += 4) {
            float rd[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) rd[u] = token(tt + u);
#pragma unroll
            for (int u = 0; u < 4; ++u) rd_s[(tt + u) * CD_THREADS + threadIdx.x] = rd[u];      // [token][group][column]
        }
        for (; tt < nt; ++tt) rd_s[tt * CD_THREADS + threadIdx.x] = token(tt);
        __syncthreads();     // (also: everyone is done with this buffer before the chunk after next is copied into it)
        {
            tt = grp;      // (as many tokens a chunk as groups)
            if (tt < nt && live) {
                float s = 0.f;
#pragma unroll
                for (int g = 0; g < CD_GROUPS; ++g) s += rd_s[tt * CD_THREADS + g * CD_COLS + col];
                a.out[(long)(c0 + tt) * a.ldo + (long)h * a.V + col0 + col] = s * a.q_scale;
            }
        }
        // (the next chunk writes rd_s behind the barrier that follows its wait)
    }
    fx_pdl_trigger();
    if (live) {
#pragma unroll
        for (int i = 0; i < RPL; ++i) {
            const int row = grp * RPL + i;
            if (row < D) sp[row * a.row_stride] = S[i];
        }
    }
}
static_assert(CD_CH == CD_GROUPS, "a chunk's read-outs are added up by one group of threads a token");

template <int RPL, bool FIXED>
int launch_cd(const CdArgs& a, int n_entries, cudaStream_t s)
{
    constexpr int DP = RPL * CD_GROUPS;
    const size_t smem = ((size_t)2 * CD_CH * ((FIXED ? 2 : 3) * DP + CD_COLS) + CD_CH * CD_THREADS) * sizeof(float);
    auto kern = channel_decay_scan_kernel<RPL, FIXED>;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    dim3 grid(n_entries, a.H, (unsigned)fx_cdiv(a.V, CD_COLS));
    // a prompt's recurrence starts on an empty device (see fx_launch_pdl_if); a decode step's is set up early
    fx_launch_pdl_if(a.n_tokens < 8 * n_entries, kern, grid, dim3(CD_THREADS), smem, s, a);
    return fx_launch_status();
}

template <bool FIXED>
int scan_for(const CdArgs& a, int n_entries, cudaStream_t s)
{
    if (a.D <= 4 * CD_GROUPS) return launch_cd<4, FIXED>(a, n_entries, s);
    if (a.D <= 8 * CD_GROUPS) return launch_cd<8, FIXED>(a, n_entries, s);
    if (a.D <= 12 * CD_GROUPS) return launch_cd<12, FIXED>(a, n_entries, s);
    return launch_cd<16, FIXED>(a, n_entries, s);
}

template <typename T>
__global__ void silu_rows_kernel(const T* __restrict__ x, long ldx, float* __restrict__ out, long ldo, int n)
{
    fx_pdl_wait();
    const T* r = x + (long)blockIdx.x * ldx;
    float* o = out + (long)blockIdx.x * ldo;
    constexpr int N = Pack<T>::N;
    if (n % N == 0 && (uintptr_t)r % 16 == 0 && (uintptr_t)o % 16 == 0) {
        for (int i = (blockIdx.y * blockDim.x + threadIdx.x) * N; i < n; i += gridDim.y * blockDim.x * N) {
            float v[N];
            Pack<T>::load(r + i, v);
#pragma unroll
            for (int e = 0; e < N; ++e) v[e] = v[e] / (1.0f + expf(-v[e]));
#pragma unroll
            for (int e = 0; e < N; e += 4) Pack<float>::store(o + i + e, v + e);
        }
        return;
    }
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < n; i += gridDim.y * blockDim.x) {
        const float v = to_f32(r[i]);
        o[i] = v / (1.0f + expf(-v));
    }
}

}  // namespace

extern "C" int fx_channel_decay_prep(const float* low, long ldl, const void* w2, int w2_dtype, const void* bias, int b_dtype,
                                     float inv_tau, float* alpha, int n_tokens, int channels, int rank, void* stream)
{
    if (n_tokens <= 0) return FX_OK;
    if (channels <= 0 || rank <= 0) return FX_ERR_SIZE;
    dim3 grid((unsigned)fx_cdiv(n_tokens, CP_TOKENS), (unsigned)fx_cdiv(channels, CP_THREADS));
    fx_launch_pdl(channel_decay_prep_kernel, grid, CP_THREADS, 0, (cudaStream_t)stream, low, ldl, w2, w2_dtype, bias, b_dtype,
                  inv_tau, alpha, n_tokens, channels, rank);
    return fx_launch_status();
}

extern "C" int fx_channel_decay_scan(const float* q, long ldq, const float* k, long ldk, const float* v, long ldv,
                                     const float* alpha, float q_scale, float* state, float* out, long ldo,
                                     const int* token_seq, const int* seq_slot, int n_tokens, int n_entries, int H, int D,
                                     int V, void* stream)
{
    if (n_tokens <= 0 || n_entries <= 0) return FX_OK;
    if (H <= 0 || H > 65535 || D <= 0 || V <= 0 || D > CD_MAX_D) return FX_ERR_SIZE;
    CdArgs a;
    a.src[0] = q; a.src[1] = k; a.src[2] = alpha; a.ld[0] = ldq; a.ld[1] = ldk; a.ld[2] = (long)H * D;
    a.v = v; a.ldv = ldv; a.q_scale = q_scale; a.decay = nullptr; a.state = state; a.row_stride = V; a.col_stride = 1;
    a.out = out; a.ldo = ldo;
    a.token_seq = token_seq; a.seq_slot = seq_slot; a.n_tokens = n_tokens; a.H = H; a.D = D; a.V = V;
    a.vec = D % 4 == 0 && ldq % 4 == 0 && ldk % 4 == 0;
    for (int i = 0; i < 3; ++i) a.vec = a.vec && (uintptr_t)a.src[i] % 16 == 0;
    return scan_for<false>(a, n_entries, (cudaStream_t)stream);
}

extern "C" int fx_fixed_decay_scan(const float* q, long ldq, const float* k, long ldk, const float* v, long ldv,
                                   const float* decay, float* state, float* out, long ldo, const int* token_seq,
                                   const int* seq_slot, int n_tokens, int n_entries, int H, int D, int V, void* stream)
{
    if (n_tokens <= 0 || n_entries <= 0) return FX_OK;
    if (H <= 0 || H > 65535 || D <= 0 || V <= 0 || D > CD_MAX_D) return FX_ERR_SIZE;
    CdArgs a;
    a.src[0] = q; a.src[1] = k; a.src[2] = nullptr; a.ld[0] = ldq; a.ld[1] = ldk; a.ld[2] = 0;
    a.v = v; a.ldv = ldv; a.q_scale = 1.f; a.decay = decay; a.state = state; a.row_stride = 1; a.col_stride = D;
    a.out = out; a.ldo = ldo;
    a.token_seq = token_seq; a.seq_slot = seq_slot; a.n_tokens = n_tokens; a.H = H; a.D = D; a.V = V;
    a.vec = D % 4 == 0 && ldq % 4 == 0 && ldk % 4 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)k % 16 == 0;
    return scan_for<true>(a, n_entries, (cudaStream_t)stream);
}

extern "C" int fx_silu_rows(const void* x, int dtype, long ldx, float* out, long ldo, int n_rows, int n, void* stream)
{
    if (n_rows <= 0 || n <= 0) return FX_OK;
    long by = fx_cdiv(n, 256 * 8);
    if (by > 64) by = 64;
    dim3 grid(n_rows, (unsigned)by);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == FX_F32) fx_launch_pdl(silu_rows_kernel<float>, grid, 256, 0, s, (const float*)x, ldx, out, ldo, n);
    else if (dtype == FX_BF16) fx_launch_pdl(silu_rows_kernel<bf16>, grid, 256, 0, s, (const bf16*)x, ldx, out, ldo, n);
    else return FX_ERR_DTYPE;
    return fx_launch_status();
}
