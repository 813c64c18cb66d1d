// The selective scan (a diagonal state-space recurrence whose step size and in/out projections depend on the token), for any
// split of a sequence into steps.  Per channel c and state n, with dt = softplus(low-rank product + bias) per token and channel,
//     S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n          y_c = sum_n S[c, n] C_n + D_c u_c          out = y * silu(z)
// A is negative, [channels, states]; B and C are one row of states per token that all channels share; u is the output of a short
// convolution and z a gate branch.  Step sizes, decays, state and read-out are 32-bit in every run.
//
// A thread owns four consecutive states of one channel, the slices of a channel are adjacent lanes, and a CTA of 128 threads takes
// 128 / slices channels of one request.  The kernel is bound by the exponentials (one per state and token; the unit does 16 a
// clock and SM) as long as nothing else shows, so a run of TB tokens is taken in phases: all its decays and inputs first (independent
// of each other), then the chain of the state (two multiply-adds a token), then the read-outs of the whole run reduced over the
// slices at once.  The lanes of a channel share what belongs to a token and channel alone: each loads the step sizes, inputs
// and gates of its share of the run's tokens, evaluates them, and finishes those tokens' outputs.  B and C, which all channels
// share, go through two buffers of shared memory (one barrier per run); all of the next run's values travel into registers
// while this one is computed.  A state row is [channels][padded states].
//
// Long prompts in parts.  The decay over a part is exp(A * sum of dt), so what a part adds to the state needs no other part:
// with ``parts`` > 1 the kernel runs twice over requests x parts.  Mode 1 walks every part but a request's last from a zero
// state without reading out and leaves that sum and the part's summed step sizes in scratch (the unit of the last part copies
// the request's state row there meanwhile, so that the second launch reads nothing that it also writes).  Mode 0 builds each
// part's first state from those, walks the part with read-out, and the request's last part writes the state row.
// The last unit of a request also moves the short convolution's last inputs into their state row (that kernel ran before).
#include "common.cuh"
#include <math.h>
using namespace ttie;

namespace {

constexpr int NT = 128, TB = 8, KPT = 4;    // threads of a CTA; tokens of a run; states of a thread
constexpr int DIRECT_TOKENS = 2;            // a request that brings this few tokens (decoded ones) is walked straight from global memory
constexpr int PART_MIN_TOKENS = 64;

__device__ __forceinline__ int slot_row_(int slot, int num_rows) { return slot < 0 ? num_rows - 1 : slot; }
// The step of a state, S <- exp(dt A) S + du B.
// A slow state (dt * A near 0) lives for thousands of tokens, and the rounding of a factor just below 1 repeats itself with every
// token: a 32-bit run adds expm1(dt * A) S + du B to S instead, which leaves only the sum's own rounding.  A bfloat16 run uses the
// hardware's 2^x on A * log2(e), which the thread then holds for A (relative error about 2^-22, far below the rounding of the
// bfloat16 operands around it).
__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
// softplus and silu: the library's accurate functions in a 32-bit run; else the hardware's exponential, logarithm and reciprocal
// (relative error about 1e-6 as well: log(1 + e) of a small e, where 1 + e has lost its digits, by the series e - e^2/2 + e^3/3).
template <typename T> struct Act {
    static __device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
    static __device__ __forceinline__ float silu(float x) { return x / (1.0f + expf(-x)); }
};
template <> struct Act<__nv_bfloat16> {
    static __device__ __forceinline__ float softplus(float x) {
        const float e = __expf(-fabsf(x));
        const float small = e * fmaf(e, fmaf(e, 0.33333334f, -0.5f), 1.0f);
        return fmaxf(x, 0.f) + (e < 0.01f ? small : __logf(1.0f + e));
    }
    static __device__ __forceinline__ float silu(float x) { return __fdividef(x, 1.0f + __expf(-x)); }
};
template <typename T> struct Decay {
    static __device__ __forceinline__ float hold(float a) { return a; }
    static __device__ __forceinline__ float of(float dt, float a) { return expm1f(dt * a); }
    static __device__ __forceinline__ float step(float e, float S, float x) { return S + fmaf(e, S, x); }
};
template <> struct Decay<__nv_bfloat16> {
    static __device__ __forceinline__ float hold(float a) { return a * 1.4426950408889634f; }
    static __device__ __forceinline__ float of(float dt, float a) { return ex2(dt * a); }
    static __device__ __forceinline__ float step(float e, float S, float x) { return fmaf(e, S, x); }
};

struct SelArgs {
    const void* u; long long ld_u;                                    // [T, I] compute dtype
    const float* dt; long long ld_dt; const float* dt_bias;           // [T, I] before bias and softplus, [I]
    const float* A; const float* D;                                   // [I, Np], [I]
    const void* bc; long long ld_bc; int col_b, col_c;                // rows that hold B and C at these columns, compute dtype
    const void* z; long long ld_z;                                    // [T, I] compute dtype
    float* state; int state_rows;                                     // [rows, I, Np]
    const void* xin; long long ld_x; float* tail; int tail_rows, taps; // the convolution's inputs [T, I] and its state rows [rows, taps - 1, I]
    const int* qsl; const int* slot_ids;
    void* out;                                                        // [T, I] compute dtype
    int I, N, Np;
    float* scratch; float* scratch_dt; int parts, mode;               // [requests * parts, I, Np], [requests * parts, I]
};

template <int SL> __device__ __forceinline__ float slices_sum(float v) {
#pragma unroll
    for (int o = 1; o < SL; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Sums over the SL adjacent lanes of a channel of CNT values per lane at once (the read-outs of a run of tokens): at every step
// a lane hands half of its values to the partner and adds the partner's other half to the half it keeps; once a lane is down to
// one value the remaining steps are butterfly additions.  Afterwards v[0 ..] holds the totals of tokens slice * CNT / SL ..
template <int O, int CNT>
__device__ __forceinline__ void run_reduce(float* v, int slice) {
    if constexpr (O >= 1) {
        if constexpr (CNT > 1) {
            constexpr int HALF = CNT / 2;
            const bool upper = (slice & O) != 0;
#pragma unroll
            for (int i = 0; i < HALF; ++i) {
                const float send = upper ? v[i] : v[i + HALF];
                const float keep = upper ? v[i + HALF] : v[i];
                v[i] = keep + __shfl_xor_sync(0xffffffffu, send, O);
            }
            run_reduce<O / 2, HALF>(v, slice);
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], O);
            run_reduce<O / 2, 1>(v, slice);
        }
    }
}
__device__ __forceinline__ void ld4(const float* p, float* o) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    o[0] = x.x; o[1] = x.y; o[2] = x.z; o[3] = x.w;
}

// Walks n tokens.  READ: with read-out (writes out); without, only the state moves.  Returns the sum of the step sizes.
template <typename T, int SL, bool READ>
__device__ __forceinline__ float walk(const SelArgs& a, int t0, int n, int c, bool cv, int slice, const float (&A)[KPT], float (&S)[KPT], float* smem) {
    constexpr int NP = SL * KPT, PC = TB / SL > 0 ? TB / SL : 1, SAME = SL / TB > 0 ? SL / TB : 1, PB = (TB * NP + NT - 1) / NT;
    const int cc = cv ? c : 0, n0 = slice * KPT;
    const T* up = reinterpret_cast<const T*>(a.u) + (size_t)t0 * a.ld_u + cc;
    const T* zp = reinterpret_cast<const T*>(a.z) + (size_t)t0 * a.ld_z + cc;
    const T* bp = reinterpret_cast<const T*>(a.bc) + (size_t)t0 * a.ld_bc + a.col_b;
    const T* cp = reinterpret_cast<const T*>(a.bc) + (size_t)t0 * a.ld_bc + a.col_c;
    const float* dp = a.dt + (size_t)t0 * a.ld_dt + cc;
    T* op = reinterpret_cast<T*>(a.out) + (size_t)t0 * a.I + cc;
    const float bias = a.dt_bias[cc], Dc = a.D[cc];
    float sum_dt = 0.f;
    if (n <= DIRECT_TOKENS) {
        for (int tt = 0; tt < n; ++tt) {
            const float dt = Act<T>::softplus(dp[(size_t)tt * a.ld_dt] + bias), u = to_f32(up[(size_t)tt * a.ld_u]), du = dt * u;
            float acc = 0.f;
#pragma unroll
            for (int i = 0; i < KPT; ++i) {
                const bool in = n0 + i < a.N;
                S[i] = Decay<T>::step(Decay<T>::of(dt, A[i]), S[i], du * (in ? to_f32(bp[(size_t)tt * a.ld_bc + n0 + i]) : 0.f));
                acc = fmaf(S[i], READ && in ? to_f32(cp[(size_t)tt * a.ld_bc + n0 + i]) : 0.f, acc);
            }
            sum_dt += dt;
            if (!READ) continue;
            acc = slices_sum<SL>(acc);
            if (slice == 0 && cv) op[(size_t)tt * a.I] = from_f32<T>(fmaf(Dc, u, acc) * Act<T>::silu(to_f32(zp[(size_t)tt * a.ld_z])));
        }
        return sum_dt;
    }
    // the lanes of a channel share the tokens of a run: lane `slice` holds step size, input and gate of tokens own .. own + PC - 1
    // (with more slices than tokens, SAME lanes hold the same one)
    const int own = slice / SAME * PC;
    float d_next[PC], d[PC], u[PC], b_next[PB], c_next[PB];
    T u_next[PC], z_next[PC], z[PC];
    auto fetch = [&](int r0, int nb) {
#pragma unroll
        for (int j = 0; j < PC; ++j) {
            const int tt = own + j;
            const bool ok = tt < nb;
            d_next[j] = ok ? dp[(size_t)(r0 + tt) * a.ld_dt] : 0.f;
            u_next[j] = ok ? up[(size_t)(r0 + tt) * a.ld_u] : from_f32<T>(0.f);
            if (READ) z_next[j] = ok ? zp[(size_t)(r0 + tt) * a.ld_z] : from_f32<T>(0.f);
        }
#pragma unroll
        for (int i = 0; i < PB; ++i) {
            const int e = i * NT + threadIdx.x, tt = e / NP, k = e - tt * NP;
            const bool ok = tt < nb && k < a.N;
            b_next[i] = ok ? to_f32(bp[(size_t)(r0 + tt) * a.ld_bc + k]) : 0.f;
            if (READ) c_next[i] = ok ? to_f32(cp[(size_t)(r0 + tt) * a.ld_bc + k]) : 0.f;
        }
    };
    auto settle = [&](int buf, int nb) {                             // what has arrived becomes the current run
        float* bs = smem + buf * 2 * TB * NP;
#pragma unroll
        for (int i = 0; i < PB; ++i) {
            const int e = i * NT + threadIdx.x;
            if (e < TB * NP) { bs[e] = b_next[i]; if (READ) bs[TB * NP + e] = c_next[i]; }
        }
#pragma unroll
        for (int j = 0; j < PC; ++j) {                               // (a token behind the last one: step size 0, which moves nothing)
            d[j] = own + j < nb ? Act<T>::softplus(d_next[j] + bias) : 0.f;
            u[j] = to_f32(u_next[j]);
            if (READ) z[j] = z_next[j];
        }
        __syncthreads();
    };
    fetch(0, min(TB, n));
    settle(0, min(TB, n));
    for (int r0 = 0, it = 0; r0 < n; r0 += TB, ++it) {
        const int nb = min(TB, n - r0);
        const bool more = r0 + TB < n;
        if (more) fetch(r0 + TB, min(TB, n - r0 - TB));
        const float* bs = smem + (it & 1) * 2 * TB * NP + n0;
        float e[TB][KPT], x[TB][KPT], y[TB];
#pragma unroll
        for (int tt = 0; tt < TB; ++tt) {
            float dt = d[tt % PC], du = d[tt % PC] * u[tt % PC], b[KPT];
            if (SL > 1) {
                dt = __shfl_sync(0xffffffffu, dt, tt / PC * SAME, SL);
                du = __shfl_sync(0xffffffffu, du, tt / PC * SAME, SL);
            }
            ld4(bs + tt * NP, b);
#pragma unroll
            for (int i = 0; i < KPT; ++i) { e[tt][i] = Decay<T>::of(dt, A[i]); x[tt][i] = du * b[i]; }
            if (!READ) sum_dt += dt;
        }
#pragma unroll
        for (int tt = 0; tt < TB; ++tt) {
#pragma unroll
            for (int i = 0; i < KPT; ++i) S[i] = Decay<T>::step(e[tt][i], S[i], x[tt][i]);
            if (READ) {
                float q[KPT];
                ld4(bs + TB * NP + tt * NP, q);
                y[tt] = fmaf(S[0], q[0], S[1] * q[1]) + fmaf(S[2], q[2], S[3] * q[3]);
            }
        }
        if (READ) {
            run_reduce<SL / 2, TB>(y, slice);
            if (cv && slice % SAME == 0) {
#pragma unroll
                for (int j = 0; j < PC; ++j)
                    if (own + j < nb) op[(size_t)(r0 + own + j) * a.I] = from_f32<T>(fmaf(Dc, u[j], y[j]) * Act<T>::silu(to_f32(z[j])));
            }
        }
        if (more) settle((it & 1) ^ 1, min(TB, n - r0 - TB));
    }
    return sum_dt;
}

template <typename T, int SL>
__global__ void __launch_bounds__(NT) selective_scan_kernel(const SelArgs a) {
    pdl_wait();                                                      // (the successor is let in at the end: its waiting CTAs would sit on the SMs of a long, latency-bound walk)
    constexpr int CH = NT / SL, NP = SL * KPT;                       // channels per CTA, padded states
    __shared__ __align__(16) float smem[4 * TB * NP];                // two buffers of B and C
    const int s = blockIdx.y / a.parts, p = blockIdx.y - s * a.parts;
    const int q0 = a.qsl[s], n = a.qsl[s + 1] - q0;
    int L = n, p_last = 0;                                           // tokens of a part, the part of the request's last token
    if (a.parts > 1 && n > 0) {
        L = max(PART_MIN_TOKENS, ((n + a.parts - 1) / a.parts + TB - 1) / TB * TB);
        p_last = (n - 1) / L;                                        // (< parts)
    }
    const bool local = a.mode == 1;
    const bool copies = local && p_last > 0 && p == a.parts - 1;     // (never a part that mode 1 walks: those lie before p_last)
    if (n <= 0 || (local ? (p >= p_last && !copies) : p > p_last)) return;
    const int slice = threadIdx.x % SL, c0 = blockIdx.x * CH, c = c0 + threadIdx.x / SL;
    const bool cv = c < a.I;
    const int cc = cv ? c : 0, n0 = slice * KPT;
    float* sp = a.state + ((size_t)slot_row_(a.slot_ids[s], a.state_rows) * a.I + cc) * NP + n0;
    auto scratch_at = [&](int part) { return a.scratch + (((size_t)s * a.parts + part) * a.I + cc) * NP + n0; };
    if (copies) {
        if (cv) *reinterpret_cast<float4*>(scratch_at(p)) = *reinterpret_cast<const float4*>(sp);
        return;
    }
    float A[KPT], S[KPT] = {0.f, 0.f, 0.f, 0.f}, sum_dt;
    ld4(a.A + (size_t)cc * NP + n0, A);
#pragma unroll
    for (int i = 0; i < KPT; ++i) A[i] = Decay<T>::hold(A[i]);
    if (local) {
        sum_dt = walk<T, SL, false>(a, q0 + p * L, min(L, n - p * L), c, cv, slice, A, S, smem);
    } else {
        ld4(p_last == 0 ? sp : scratch_at(a.parts - 1), S);          // the state row as it was before the step
        for (int j = 0; j < p; ++j) {                                // then the parts before this one: S <- exp(A * sum of dt) S + what the part adds
            float add[KPT];
            ld4(scratch_at(j), add);
            const float sdt = a.scratch_dt[((size_t)s * a.parts + j) * a.I + cc];
#pragma unroll
            for (int i = 0; i < KPT; ++i) S[i] = Decay<T>::step(Decay<T>::of(sdt, A[i]), S[i], add[i]);
        }
        walk<T, SL, true>(a, q0 + p * L, min(L, n - p * L), c, cv, slice, A, S, smem);
    }
    pdl_launch_dependents();
    if (cv && (local || p == p_last)) {
        *reinterpret_cast<float4*>(local ? scratch_at(p) : sp) = make_float4(S[0], S[1], S[2], S[3]);
        if (local && slice == 0) a.scratch_dt[((size_t)s * a.parts + p) * a.I + c] = sum_dt;
    }
    if (!local && p == p_last && a.taps > 1 && threadIdx.x < CH && c0 + (int)threadIdx.x < a.I) {
        // the convolution's last taps - 1 inputs, oldest first: those of this step, and before them what the row held
        const int ch = c0 + threadIdx.x;
        const T* x = reinterpret_cast<const T*>(a.xin) + ch;
        float* mine = a.tail + (size_t)slot_row_(a.slot_ids[s], a.tail_rows) * (a.taps - 1) * a.I + ch;
        for (int i = 0; i < a.taps - 1; ++i) {                       // ascending: row i takes from an old row behind it, or from the step
            const int idx = n - (a.taps - 1) + i;
            mine[(size_t)i * a.I] = idx >= 0 ? to_f32(x[(size_t)(q0 + idx) * a.ld_x]) : mine[(size_t)(a.taps - 1 + idx) * a.I];
        }
    }
}

int state_slices(int N) {
    int sl = 1;
    while (sl * KPT < N) sl <<= 1;
    return sl;
}
}  // namespace

// padded states of a state row (0: more states than the kernel takes)
extern "C" int ttie_selective_state_pad(int N) { return N < 1 || N > 128 ? 0 : state_slices(N) * KPT; }

// parts > 1: scratch holds requests * parts * channels * (padded states + 1) floats
extern "C" int ttie_selective_scan(const void* u, long long ld_u, const float* dt, long long ld_dt, const float* dt_bias, const float* A,
                                   const float* D, const void* bc, long long ld_bc, int col_b, int col_c, const void* z, long long ld_z,
                                   float* state, int state_rows, const void* xin, long long ld_x, float* tail, int tail_rows, int taps,
                                   const int* qsl, const int* slot_ids, int num_seqs, void* out, int I, int N, int parts, float* scratch,
                                   int dtype, void* stream) {
    if (num_seqs <= 0) return 0;
    if (N < 1 || N > 128) TTIE_FAIL("selective_scan: %d states per channel (1 to 128)", N);
    if (parts < 1 || (parts > 1 && !scratch) || (long long)num_seqs * parts > 65535)
        TTIE_FAIL("selective_scan: %d parts for %d requests", parts, num_seqs);
    if (taps > 1 && (!tail || !xin)) TTIE_FAIL("selective_scan: %d taps need state rows and inputs", taps);
    if (dtype != kF32 && dtype != kBF16) TTIE_FAIL("selective_scan: unknown dtype %d", dtype);
    SelArgs a;
    a.u = u; a.ld_u = ld_u; a.dt = dt; a.ld_dt = ld_dt; a.dt_bias = dt_bias; a.A = A; a.D = D; a.bc = bc; a.ld_bc = ld_bc; a.col_b = col_b;
    a.col_c = col_c; a.z = z; a.ld_z = ld_z; a.state = state; a.state_rows = state_rows; a.xin = xin; a.ld_x = ld_x; a.tail = tail;
    a.tail_rows = tail_rows; a.taps = taps; a.qsl = qsl; a.slot_ids = slot_ids; a.out = out; a.I = I; a.N = N;
    const int sl = state_slices(N);
    a.Np = KPT * sl; a.parts = parts; a.scratch = scratch;
    a.scratch_dt = scratch ? scratch + (size_t)num_seqs * parts * I * a.Np : nullptr;
    const dim3 grid(ceil_div(I, NT / sl), num_seqs * parts);
    cudaStream_t s = (cudaStream_t)stream;
    for (int mode = parts > 1 ? 1 : 0; mode >= 0; --mode) {          // (mode 1: every part's own sum, from a zero state)
        a.mode = mode;
#define SEL_CASE(L_)                                                                                                      \
        if (sl == L_) {                                                                                                   \
            if (dtype == kF32) TTIE_LAUNCH((selective_scan_kernel<float, L_>), grid, NT, 0, s, a);                        \
            else TTIE_LAUNCH((selective_scan_kernel<__nv_bfloat16, L_>), grid, NT, 0, s, a);                              \
        }
        SEL_CASE(1) SEL_CASE(2) SEL_CASE(4) SEL_CASE(8) SEL_CASE(16) SEL_CASE(32)
#undef SEL_CASE
        TTIE_CHECK_LAUNCH("selective_scan");
    }
    return 0;
}
