// The selective state space of a Mamba mixer: per request a state S [inner, n_state], 32-bit, and for every token
//
//   a channel's row s of it:   step = softplus(dt + bias),   s = e^(-step e^A_log) * s + step x B,   y = s . C + D x
//   out = y silu(z)                                          (B and C: one number a state, shared by the channels)
//
// Channels never meet: L lanes share a channel's states (NPL of them each, in runs of up to four, so that B and C are read
// from shared memory sixteen bytes at a time) and keep them in registers for the whole step; the tokens of a request are
// taken in order, in the same order of operations however the request was cut into steps.  A block of 128 threads takes
// 128 / L channels of one request; the tokens' rows come a chunk of them at a time, the next chunk's into registers while
// this one is worked on.  The step size, the products dt x and the skip and gate are worked out once a (token, channel),
// not by every lane; the lanes' shares of the read-out meet once a chunk, through shared memory.
//
// Everything is 32-bit arithmetic; x and z come in the engine's element type.  A state that decays slowly is multiplied a
// thousand times by numbers just below 1, so that a bias of half a unit in their last place would show: where the
// exponent is small the state moves by S (e^a - 1) with e^a - 1 from its Taylor series, whose error is relative to a.
// With x in 16 bits, whose rounding is five hundred times larger than such a bias over a thousand tokens, the hardware's
// exponential does: a third of the instructions.
#include "common.cuh"
#include "api.h"

namespace {

// z / (1 + e^-z); in 16 bits the hardware's exponential and quotient do.
template <typename T> __device__ __forceinline__ float gate_silu(float z) {
    return sizeof(T) == 2 ? __fdividef(z, 1.0f + __expf(-z)) : z / (1.0f + expf(-z));
}

// e^a S + u for a <= 0; T = bf16: a comes times log2 e.
template <typename T>
__device__ __forceinline__ float decay_add(float S, float a, float u)
{
    if (sizeof(T) == 2) {
        float e;
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(a));
        return fmaf(e, S, u);
    }
    // a > -1/8: e^a - 1 = a (1 + a/2 (1 + a/3 (1 + a/4 (1 + a/5)))), the next term below 5e-8 of the sum
    float p = fmaf(a, 1.0f / 120.0f, 1.0f / 24.0f);
    p = fmaf(p, a, 1.0f / 6.0f);
    p = fmaf(p, a, 0.5f);
    p = fmaf(p, a, 1.0f) * a;
    const float e = __expf(a);
    const bool slow = a > -0.125f;
    return fmaf(S, slow ? p : e, u) + (slow ? S : 0.f);
}

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

constexpr int SC_THREADS = 128;

template <int N> __device__ __forceinline__ void load_vec(const float* p, float* o) {
    if (N == 4) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        o[0] = v.x; o[N > 1 ? 1 : 0] = v.y; o[N > 2 ? 2 : 0] = v.z; o[N > 3 ? 3 : 0] = v.w;
    } else if (N == 2) {
        const float2 v = *reinterpret_cast<const float2*>(p);
        o[0] = v.x; o[N > 1 ? 1 : 0] = v.y;
    } else o[0] = *p;
}

struct ScArgs {
    const float* dt; long ldt; const void* dt_bias; int db_dtype;
    // (instead of dt, every entry bringing one token) rows [rank] of the small matrix, and the tokens' low-rank rows
    const void* w_dt; long ldw; int w_bf16, rank; const float* low; long ldlow;
    const void* x; long ldx; const void* z; long ldz;
    const float* bc; long ldbc;              // [tokens][B (n_state) | C (n_state)]
    const float* a_log; const float* d_skip; // [inner][n_state], [inner]
    float* state;                            // [slots, inner, n_state]
    void* out; long ldo;
    const int *token_seq, *seq_slot;
    int n_tokens, inner, n_state;
};

// STEPS: the kernel works out the step sizes itself (a.w_dt).
template <typename T, int L, int NPL, bool STEPS>
__global__ void __launch_bounds__(SC_THREADS) selective_scan_kernel(const ScArgs a)
{
    constexpr int CB = SC_THREADS / L;                       // channels a block
    constexpr int VEC = NPL < 4 ? NPL : 4;                   // states a lane holds side by side
    constexpr int NP = L * NPL;                              // states a channel, padded
    // tokens a chunk: long enough that the next chunk's rows arrive while one is worked on, as shared memory allows
    constexpr int SC_CH = L >= 8 && NP <= 64 ? 32 : 16;
    constexpr int EPT = (SC_CH * CB + SC_THREADS - 1) / SC_THREADS;     // (token, channel) pairs a thread
    constexpr int BPT = (SC_CH * NP + SC_THREADS - 1) / SC_THREADS;     // (token, state) pairs a thread
    __shared__ float dt_s[SC_CH][CB], dx_s[SC_CH][CB];
    __shared__ float x_s[SC_CH][CB], z_s[SC_CH][CB];
    __shared__ __align__(16) float b_s[SC_CH][NP], c_s[SC_CH][NP];
    __shared__ float rd_s[SC_CH][SC_THREADS];
    const int ch0 = blockIdx.y * CB, I = a.inner, N = a.n_state;
    const int cl = threadIdx.x / L, part = threadIdx.x % L, ch = ch0 + cl;
    const bool live = ch < I;
    const T* xp = reinterpret_cast<const T*>(a.x);
    const T* zp = reinterpret_cast<const T*>(a.z);

    // Weights first: they are nobody's work.  (Nothing that any kernel or copy writes is read before the wait, however long
    // ago it was written: the SM's own cache may still hold what stood there before.)
    float S[NPL], A[NPL];        // the states and their rates
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
        const int n = (i / VEC) * VEC * L + part * VEC + i % VEC;
        A[i] = live && n < N ? -expf(a.a_log[(long)ch * N + n]) * (sizeof(T) == 2 ? 1.4426950408889634f : 1.f) : 0.f;
    }
    // the channel of this thread's (token, channel) pairs is the same in every chunk: CB divides the block
    const int pc = threadIdx.x % CB, ptt = threadIdx.x / CB, pch = ch0 + pc;
    const bool plive = pch < I;
    const int gch = plive ? pch : I - 1;
    const float bias = load_any(a.dt_bias, a.db_dtype, gch), skip = a.d_skip[gch];

    // A decode step's step sizes: the low-rank row of the entry's one token times the block's rows of the small matrix,
    // which the lanes of a channel share out.
    const int row_pieces = a.rank / 8;
    uint4 wp[2];
    const bool pieces = STEPS && a.w_bf16 && a.rank % 8 == 0 && row_pieces <= 2 * L;
    if (pieces && live) {
        const uint4* wr = reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(a.w_dt) + (long)ch * a.ldw);
#pragma unroll
        for (int k = 0; k < 2; ++k)
            if (part + k * L < row_pieces) wp[k] = wr[part + k * L];
    }
    fx_pdl_wait_only();
    const int b = blockIdx.x;
    const int r0 = first_row_of(a.token_seq, a.n_tokens, b), r1 = first_row_of(a.token_seq, a.n_tokens, b + 1);
    if (r1 <= r0) return;
    float* sp = a.state + ((long)a.seq_slot[b] * I + (live ? ch : 0)) * N;
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
        const int n = (i / VEC) * VEC * L + part * VEC + i % VEC;
        S[i] = live && n < N ? sp[n] : 0.f;
    }
    if (STEPS) {
        float acc = 0.f;
        const float* lr = a.low + (long)r0 * a.ldlow;
        if (live) {
            if (pieces) {
#pragma unroll
                for (int k = 0; k < 2; ++k)
                    if (part + k * L < row_pieces) {
                        const float* l = lr + (part + k * L) * 8;
                        const uint32_t w4[4] = {wp[k].x, wp[k].y, wp[k].z, wp[k].w};
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            acc = fmaf(__uint_as_float(w4[e] << 16), l[2 * e], acc);
                            acc = fmaf(__uint_as_float(w4[e] & 0xffff0000u), l[2 * e + 1], acc);
                        }
                    }
            } else {
                for (int r = part; r < a.rank; r += L) acc = fmaf(load_any(a.w_dt, a.w_bf16 ? FX_BF16 : FX_F32, (long)ch * a.ldw + r), lr[r], acc);
            }
        }
#pragma unroll
        for (int o = L >> 1; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (part == 0) dt_s[0][cl] = acc;
        __syncthreads();
    }

    float fdt[EPT], fb[BPT], fc[BPT];
    T fx[EPT], fz[EPT];      // (as loaded: a conversion here would wait for the load)
    auto fetch = [&](int c0, int nt) {       // every load unconditional, from places clamped into the chunk
#pragma unroll
        for (int e = 0; e < EPT; ++e) {
            const long t = c0 + min(ptt + e * L, nt - 1);
            fdt[e] = STEPS ? dt_s[0][pc] : a.dt[t * a.ldt + gch];      // (STEPS: one token, one chunk)
            fx[e] = xp[t * a.ldx + gch];
            fz[e] = zp[t * a.ldz + gch];
        }
#pragma unroll
        for (int e = 0; e < BPT; ++e) {
            const int idx = threadIdx.x + e * SC_THREADS;
            const long t = c0 + min(idx / NP, nt - 1);
            const int n = min(idx % NP, N - 1);
            fb[e] = a.bc[t * a.ldbc + n];
            fc[e] = a.bc[t * a.ldbc + N + n];
        }
    };
    fetch(r0, min(SC_CH, r1 - r0));
    for (int c0 = r0; c0 < r1; c0 += SC_CH) {
        const int nt = min(SC_CH, r1 - c0);
        __syncthreads();             // the chunk before is done with the staged rows
#pragma unroll
        for (int e = 0; e < EPT; ++e) {
            const int tt = ptt + e * L;
            if (tt < SC_CH) {
                const float d = fx_softplus(fdt[e] + bias);
                const float xx = to_f32(fx[e]);
                dt_s[tt][pc] = d; dx_s[tt][pc] = d * xx;
                x_s[tt][pc] = xx; z_s[tt][pc] = to_f32(fz[e]);
            }
        }
#pragma unroll
        for (int e = 0; e < BPT; ++e) {
            const int idx = threadIdx.x + e * SC_THREADS;
            if (idx < SC_CH * NP) {
                const bool in = idx % NP < N;
                b_s[idx / NP][idx % NP] = in ? fb[e] : 0.f;
                c_s[idx / NP][idx % NP] = in ? fc[e] : 0.f;
            }
        }
        __syncthreads();
        if (c0 + SC_CH < r1) fetch(c0 + SC_CH, min(SC_CH, r1 - c0 - SC_CH));
        auto token = [&](int tt) {      // one token: the states move on; this lane's share of the read-out
            const float d = dt_s[tt][cl], dx = dx_s[tt][cl];
            float y0 = 0.f, y1 = 0.f;
#pragma unroll
            for (int i = 0; i < NPL; i += VEC) {
                float bb[VEC], cc[VEC];
                load_vec<VEC>(&b_s[tt][(i / VEC) * VEC * L + part * VEC], bb);
                load_vec<VEC>(&c_s[tt][(i / VEC) * VEC * L + part * VEC], cc);
#pragma unroll
                for (int j = 0; j < VEC; ++j) {
                    S[i + j] = decay_add<T>(S[i + j], d * A[i + j], dx * bb[j]);
                    if (j & 1) y1 = fmaf(S[i + j], cc[j], y1); else y0 = fmaf(S[i + j], cc[j], y0);
                }
            }
            return y0 + y1;
        };
        int tt0 = 0;
        for (; tt0 + 4 <= nt; tt0 += 4) {
            float rd[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) rd[u] = token(tt0 + u);
#pragma unroll
            for (int u = 0; u < 4; ++u) rd_s[tt0 + u][threadIdx.x] = rd[u];
        }
        for (; tt0 < nt; ++tt0) rd_s[tt0][threadIdx.x] = token(tt0);
        __syncthreads();
#pragma unroll
        for (int e = 0; e < EPT; ++e) {
            const int tt = ptt + e * L;
            if (tt < nt && plive) {
                float y = 0.f;
#pragma unroll
                for (int l = 0; l < L; ++l) y += rd_s[tt][pc * L + l];
                y = fmaf(skip, x_s[tt][pc], y);
                const float zz = z_s[tt][pc];
                reinterpret_cast<T*>(a.out)[(long)(c0 + tt) * a.ldo + pch] = from_f32<T>(y * gate_silu<T>(zz));
            }
        }
    }
    fx_pdl_trigger();
    if (live) {
#pragma unroll
        for (int i = 0; i < NPL; ++i) {
            const int n = (i / VEC) * VEC * L + part * VEC + i % VEC;
            if (n < N) sp[n] = S[i];
        }
    }
}

template <typename T, int L, int NPL>
int launch_sc(const ScArgs& a, int n_entries, cudaStream_t s)
{
    dim3 grid(n_entries, (unsigned)fx_cdiv(a.inner, SC_THREADS / L));
    // a prompt's recurrence starts on an empty device (see fx_launch_pdl_if); a decode step's is set up early
    if (a.w_dt) fx_launch_pdl(selective_scan_kernel<T, L, NPL, true>, grid, dim3(SC_THREADS), 0, s, a);
    else fx_launch_pdl_if(a.n_tokens < 8 * n_entries, selective_scan_kernel<T, L, NPL, false>, grid, dim3(SC_THREADS), 0, s, a);
    return fx_launch_status();
}

template <typename T>
int scan_for(const ScArgs& a, int n_entries, cudaStream_t s)
{
    const int n = a.n_state;
    // Few channels leave the schedulers with a warp each, which waits for its own results: two states a lane and twice
    // the warps then.
    if (n > 8 && n <= 16 && (long)n_entries * a.inner * 4 / 32 < 6L * fx_sm_count()) return launch_sc<T, 8, 2>(a, n_entries, s);
    if (n <= 4) return launch_sc<T, 1, 4>(a, n_entries, s);
    if (n <= 8) return launch_sc<T, 2, 4>(a, n_entries, s);
    if (n <= 16) return launch_sc<T, 4, 4>(a, n_entries, s);
    if (n <= 32) return launch_sc<T, 8, 4>(a, n_entries, s);
    if (n <= 64) return launch_sc<T, 8, 8>(a, n_entries, s);
    if (n <= 128) return launch_sc<T, 16, 8>(a, n_entries, s);
    return launch_sc<T, 32, 8>(a, n_entries, s);
}

__global__ void split_rows_kernel(const float* __restrict__ x, long ldx, bf16* __restrict__ out, long ldo, int n_tokens, int n,
                                  int pad)
{
    fx_pdl_wait();
    const long total = (long)n_tokens * pad;
    for (long idx = blockIdx.x * (long)blockDim.x + threadIdx.x; idx < total; idx += (long)gridDim.x * blockDim.x) {
        const long t = idx / pad;
        const int i = (int)(idx - t * pad);
        const float v = i < n ? x[t * ldx + i] : 0.f;
        const bf16 hi = __float2bfloat16_rn(v);
        out[t * ldo + i] = hi;
        out[t * ldo + pad + i] = __float2bfloat16_rn(v - __bfloat162float(hi));
    }
}

}  // namespace

// w_dt (optional, [inner][ldw], its first `rank` columns): dt is then w_dt . low, worked out here, `dt` being the rows low
// [tokens][rank]; only when every entry of the step brings exactly one token.
extern "C" int fx_selective_scan(const float* dt, long ldt, const void* w_dt, int w_dtype, long ldw, int rank,
                                 const void* dt_bias, int db_dtype, const void* x, long ldx,
                                 const void* z, long ldz, int dtype, const float* bc, long ldbc, const float* a_log,
                                 const float* d_skip, float* state, void* out, long ldo, const int* token_seq,
                                 const int* seq_slot, int n_tokens, int n_entries, int inner, int n_state, void* stream)
{
    if (n_tokens <= 0 || n_entries <= 0) return FX_OK;
    if (inner <= 0 || n_state <= 0 || n_state > 256 || fx_cdiv(inner, 4) > 65535) return FX_ERR_SIZE;
    if (w_dt && (n_tokens != n_entries || rank <= 0 || ldw < rank || (w_dtype == FX_BF16 && rank % 8 == 0 && (ldw % 8 || (uintptr_t)w_dt % 16))))
        return FX_ERR_SIZE;
    if (w_dt && w_dtype != FX_BF16 && w_dtype != FX_F32) return FX_ERR_DTYPE;
    ScArgs a;
    a.w_dt = w_dt; a.ldw = ldw; a.w_bf16 = w_dtype == FX_BF16; a.rank = w_dt ? rank : 0; a.low = dt; a.ldlow = ldt;
    a.dt = dt; a.ldt = ldt; a.dt_bias = dt_bias; a.db_dtype = db_dtype; a.x = x; a.ldx = ldx; a.z = z; a.ldz = ldz;
    a.bc = bc; a.ldbc = ldbc; a.a_log = a_log; a.d_skip = d_skip; a.state = state; a.out = out; a.ldo = ldo;
    a.token_seq = token_seq; a.seq_slot = seq_slot; a.n_tokens = n_tokens; a.inner = inner; a.n_state = n_state;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == FX_F32) return scan_for<float>(a, n_entries, s);
    if (dtype == FX_BF16) return scan_for<bf16>(a, n_entries, s);
    return FX_ERR_DTYPE;
}

extern "C" int fx_split_rows(const float* x, long ldx, void* out, long ldo, int n_tokens, int n, int pad, void* stream)
{
    if (n_tokens <= 0) return FX_OK;
    if (n <= 0 || pad < n) return FX_ERR_SIZE;
    long blocks = fx_cdiv((long)n_tokens * pad, 256);
    if (blocks > fx_sm_count() * 16L) blocks = fx_sm_count() * 16L;
    fx_launch_pdl(split_rows_kernel, (unsigned)blocks, 256, 0, (cudaStream_t)stream, x, ldx, (bf16*)out, ldo, n_tokens, n, pad);
    return fx_launch_status();
}
