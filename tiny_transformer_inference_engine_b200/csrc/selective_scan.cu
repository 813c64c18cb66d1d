// The selective scan (a diagonal state-space recurrence whose step size and in/out projections depend on the token), for any
// split of a sequence into steps.  Per channel c and state n, with dt = softplus(low-rank product + bias) per token and channel,
//     S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n          y_c = sum_n S[c, n] C_n + D_c u_c          out = y * silu(z)
// A is negative, [channels, states]; B and C are one row of states per token that all channels share; u is the output of a short
// convolution and z a gate branch.  Step sizes, decays, state and read-out are 32-bit in every run.
//
// A thread owns KPT consecutive states of one channel (4 for up to 128 states, 8 up to 256, 16 up to 512), the lanes of a
// channel's slices adjacent, so the read-out is a few shuffles; a CTA of 128 threads takes 128 / slices channels of one
// request.  A state row is [channels][padded states].  The step's tokens of a request are walked in order, a run of them at a
// time: while one run is computed the next one's rows travel into registers; step sizes are evaluated once per token and
// channel on the way into shared memory, and the read-outs leave through shared memory in whole rows.
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

constexpr int NT = 128;
constexpr int DIRECT_TOKENS = 2;            // a request that brings this few tokens (decoded ones) is walked straight from global memory
constexpr int PART_MIN_TOKENS = 64;

__device__ __forceinline__ int slot_row_(int slot, int num_rows) { return slot < 0 ? num_rows - 1 : slot; }
__device__ __forceinline__ float softplusf_(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float siluf_(float x) { return x / (1.0f + expf(-x)); }

// One step S <- exp(dt * A) S + x.  A slow state (dt * A near 0) lives for thousands of tokens, and the rounding of a factor just
// below 1 repeats itself with every token: a 32-bit run adds expm1(dt * A) S + x to S instead, which leaves only the sum's own
// rounding.  A bfloat16 run uses the hardware's 2^x on A * log2(e), which the thread then holds for A (relative error about
// 2^-22, far below the rounding of the bfloat16 operands around it).
template <typename T> struct Decay {
    static __device__ __forceinline__ float hold(float a) { return a; }
    static __device__ __forceinline__ float step(float dt, float a, float S, float x) { return S + fmaf(expm1f(dt * a), S, x); }
};
template <> struct Decay<__nv_bfloat16> {
    static __device__ __forceinline__ float hold(float a) { return a * 1.4426950408889634f; }
    static __device__ __forceinline__ float step(float dt, float a, float S, float x) {
        float y;
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(dt * a));
        return fmaf(y, S, x);
    }
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

template <typename T, int KPT, int SL>
__global__ void __launch_bounds__(NT) selective_scan_kernel(const SelArgs a) {
    pdl_wait();                                                      // (the successor is let in at the end: its waiting CTAs would sit on the SMs of a long, latency-bound walk)
    constexpr int TB = 64 / KPT, CH = NT / SL, NP = SL * KPT;        // tokens per run, channels per CTA, padded states
    constexpr int PC = (TB * CH + NT - 1) / NT, PB = (TB * NP + NT - 1) / NT;
    __shared__ __align__(16) float b_s[TB][NP], c_s[TB][NP];
    __shared__ float dt_s[TB][CH], u_s[TB][CH], z_s[TB][CH], y_s[TB][CH + 1];
    const int s = blockIdx.y / a.parts, p = blockIdx.y - s * a.parts;
    int t0 = a.qsl[s], n = a.qsl[s + 1] - t0;
    const int q0 = t0, n_all = n;
    int L = n, p_last = 0;                                           // tokens of a part, the part of the request's last token
    if (a.parts > 1 && n > 0) {
        L = max(PART_MIN_TOKENS, ((n + a.parts - 1) / a.parts + 15) / 16 * 16);
        p_last = (n - 1) / L;                                        // (< parts)
    }
    const bool local = a.mode == 1;
    const bool copies = local && p_last > 0 && p == a.parts - 1;     // (never a part that mode 1 walks: those lie before p_last)
    if (n <= 0 || (local ? (p >= p_last && !copies) : p > p_last)) return;
    const int slice = threadIdx.x % SL, cl = threadIdx.x / SL;
    const int c0 = blockIdx.x * CH, c = c0 + cl;
    const bool cv = c < a.I;
    const int cc = cv ? c : 0, n0 = slice * KPT;
    const size_t srow = slot_row_(a.slot_ids[s], a.state_rows);
    float* sp = a.state + (srow * a.I + cc) * NP + n0;
    auto scratch_at = [&](int part) { return a.scratch + (((size_t)s * a.parts + part) * a.I + cc) * NP + n0; };
    if (copies) {
        if (cv)
#pragma unroll
            for (int i = 0; i < KPT; i += 4) *reinterpret_cast<float4*>(scratch_at(p) + i) = *reinterpret_cast<const float4*>(sp + i);
        return;
    }
    float Ah[KPT], S[KPT];
#pragma unroll
    for (int i = 0; i < KPT; i += 4) {
        const float4 x = *reinterpret_cast<const float4*>(a.A + (size_t)cc * NP + n0 + i);
        Ah[i] = Decay<T>::hold(x.x); Ah[i + 1] = Decay<T>::hold(x.y); Ah[i + 2] = Decay<T>::hold(x.z); Ah[i + 3] = Decay<T>::hold(x.w);
    }
#pragma unroll
    for (int i = 0; i < KPT; ++i) S[i] = 0.f;
    if (!local) {
        const float* src = p_last == 0 ? sp : scratch_at(a.parts - 1);      // the state row as it was before the step
#pragma unroll
        for (int i = 0; i < KPT; i += 4) {
            const float4 x = *reinterpret_cast<const float4*>(src + i);
            S[i] = x.x; S[i + 1] = x.y; S[i + 2] = x.z; S[i + 3] = x.w;
        }
        for (int j = 0; j < p; ++j) {                                // then the parts before this one
            const float sdt = a.scratch_dt[((size_t)s * a.parts + j) * a.I + cc];
            const float* add = scratch_at(j);
#pragma unroll
            for (int i = 0; i < KPT; i += 4) {
                const float4 x = *reinterpret_cast<const float4*>(add + i);
                S[i] = Decay<T>::step(sdt, Ah[i], S[i], x.x); S[i + 1] = Decay<T>::step(sdt, Ah[i + 1], S[i + 1], x.y);
                S[i + 2] = Decay<T>::step(sdt, Ah[i + 2], S[i + 2], x.z); S[i + 3] = Decay<T>::step(sdt, Ah[i + 3], S[i + 3], x.w);
            }
        }
    }
    t0 += p * L;
    n = min(L, n - p * L);
    const T* up = reinterpret_cast<const T*>(a.u) + (size_t)t0 * a.ld_u;
    const T* zp = reinterpret_cast<const T*>(a.z) + (size_t)t0 * a.ld_z;
    const T* bp = reinterpret_cast<const T*>(a.bc) + (size_t)t0 * a.ld_bc + a.col_b;
    const T* cp = reinterpret_cast<const T*>(a.bc) + (size_t)t0 * a.ld_bc + a.col_c;
    const float* dp = a.dt + (size_t)t0 * a.ld_dt;
    T* op = reinterpret_cast<T*>(a.out) + (size_t)t0 * a.I;
    float sum_dt = 0.f;
    if (n <= DIRECT_TOKENS) {
        const float bias = a.dt_bias[cc], Dc = a.D[cc];
        for (int tt = 0; tt < n; ++tt) {
            const float dt = softplusf_(dp[(size_t)tt * a.ld_dt + cc] + bias), u = to_f32(up[(size_t)tt * a.ld_u + cc]), du = dt * u;
            float acc = 0.f;
#pragma unroll
            for (int i = 0; i < KPT; ++i) {
                const bool in = n0 + i < a.N;
                S[i] = Decay<T>::step(dt, Ah[i], S[i], du * (in ? to_f32(bp[(size_t)tt * a.ld_bc + n0 + i]) : 0.f));
                acc = fmaf(S[i], (in && !local) ? to_f32(cp[(size_t)tt * a.ld_bc + n0 + i]) : 0.f, acc);
            }
            sum_dt += dt;
            if (local) continue;
            acc = slices_sum<SL>(acc);
            if (slice == 0 && cv) op[(size_t)tt * a.I + c] = from_f32<T>(fmaf(Dc, u, acc) * siluf_(to_f32(zp[(size_t)tt * a.ld_z + c])));
        }
    } else {
        // this thread's share of a run: elements e = i * NT + thread of [tokens][channels], always the same channel
        const int lc = threadIdx.x % CH, lt = threadIdx.x / CH, lch = c0 + lc;
        const bool lcv = lch < a.I;
        const float lbias = lcv ? a.dt_bias[lch] : 0.f, lD = lcv ? a.D[lch] : 0.f;
        constexpr int TSTEP = NT / CH;                               // tokens between a thread's elements
        float dreg[PC], breg[PB], creg[PB];
        T ureg[PC], zreg[PC];
        auto fetch = [&](int r0, int nb) {
#pragma unroll
            for (int i = 0; i < PC; ++i) {
                const int tt = lt + i * TSTEP;
                const bool ok = tt < nb && lcv;
                dreg[i] = ok ? dp[(size_t)(r0 + tt) * a.ld_dt + lch] : 0.f;
                ureg[i] = ok ? up[(size_t)(r0 + tt) * a.ld_u + lch] : from_f32<T>(0.f);
                zreg[i] = (ok && !local) ? zp[(size_t)(r0 + tt) * a.ld_z + lch] : from_f32<T>(0.f);
            }
#pragma unroll
            for (int i = 0; i < PB; ++i) {
                const int e = i * NT + threadIdx.x, tt = e / NP, k = e - tt * NP;
                const bool ok = tt < nb && k < a.N;
                breg[i] = ok ? to_f32(bp[(size_t)(r0 + tt) * a.ld_bc + k]) : 0.f;
                creg[i] = (ok && !local) ? to_f32(cp[(size_t)(r0 + tt) * a.ld_bc + k]) : 0.f;
            }
        };
        fetch(0, min(TB, n));
        for (int r0 = 0; r0 < n; r0 += TB) {
            const int nb = min(TB, n - r0);
#pragma unroll
            for (int i = 0; i < PC; ++i) {
                const int tt = lt + i * TSTEP;
                if (tt < nb) {
                    dt_s[tt][lc] = softplusf_(dreg[i] + lbias);
                    u_s[tt][lc] = to_f32(ureg[i]);
                    z_s[tt][lc] = to_f32(zreg[i]);
                }
            }
#pragma unroll
            for (int i = 0; i < PB; ++i) {
                const int e = i * NT + threadIdx.x, tt = e / NP, k = e - tt * NP;
                if (tt < TB) { b_s[tt][k] = breg[i]; c_s[tt][k] = creg[i]; }
            }
            __syncthreads();
            if (r0 + TB < n) fetch(r0 + TB, min(TB, n - r0 - TB));
#pragma unroll
            for (int tt = 0; tt < TB; ++tt) {
                if (tt < nb) {                                       // (the same for every thread of the CTA)
                    const float dt = dt_s[tt][cl], du = dt * u_s[tt][cl];
                    float acc = 0.f;
#pragma unroll
                    for (int i = 0; i < KPT; i += 4) {
                        const float4 b = *reinterpret_cast<const float4*>(&b_s[tt][n0 + i]);
                        S[i] = Decay<T>::step(dt, Ah[i], S[i], du * b.x); S[i + 1] = Decay<T>::step(dt, Ah[i + 1], S[i + 1], du * b.y);
                        S[i + 2] = Decay<T>::step(dt, Ah[i + 2], S[i + 2], du * b.z); S[i + 3] = Decay<T>::step(dt, Ah[i + 3], S[i + 3], du * b.w);
                        if (!local) {                                // (the same for every thread of the grid)
                            const float4 q = *reinterpret_cast<const float4*>(&c_s[tt][n0 + i]);
                            acc = fmaf(S[i], q.x, acc); acc = fmaf(S[i + 1], q.y, acc); acc = fmaf(S[i + 2], q.z, acc); acc = fmaf(S[i + 3], q.w, acc);
                        }
                    }
                    if (local) { sum_dt += dt; continue; }
                    acc = slices_sum<SL>(acc);
                    if (slice == 0) y_s[tt][cl] = acc;
                }
            }
            __syncthreads();
            if (!local) {
#pragma unroll
                for (int i = 0; i < PC; ++i) {
                    const int tt = lt + i * TSTEP;
                    if (tt < nb && lcv) op[(size_t)(r0 + tt) * a.I + lch] = from_f32<T>(fmaf(lD, u_s[tt][lc], y_s[tt][lc]) * siluf_(z_s[tt][lc]));
                }
                __syncthreads();
            }
        }
    }
    pdl_launch_dependents();
    if (cv && (local || p == p_last)) {
        float* dst = local ? scratch_at(p) : sp;
#pragma unroll
        for (int i = 0; i < KPT; i += 4) *reinterpret_cast<float4*>(dst + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
        if (local && slice == 0) a.scratch_dt[((size_t)s * a.parts + p) * a.I + c] = sum_dt;
    }
    if (!local && p == p_last && a.taps > 1 && threadIdx.x < CH && c0 + (int)threadIdx.x < a.I) {
        // the convolution's last taps - 1 inputs, oldest first: those of this step, and before them what the row held
        const int ch = c0 + threadIdx.x;
        const T* x = reinterpret_cast<const T*>(a.xin) + ch;
        float* mine = a.tail + (size_t)slot_row_(a.slot_ids[s], a.tail_rows) * (a.taps - 1) * a.I + ch;
        for (int i = 0; i < a.taps - 1; ++i) {                       // ascending: row i takes from an old row behind it, or from the step
            const int idx = n_all - (a.taps - 1) + i;
            mine[(size_t)i * a.I] = idx >= 0 ? to_f32(x[(size_t)(q0 + idx) * a.ld_x]) : mine[(size_t)(a.taps - 1 + idx) * a.I];
        }
    }
}

int states_per_thread(int N) { return N <= 128 ? 4 : N <= 256 ? 8 : 16; }
int state_slices(int N) {
    const int k = states_per_thread(N);
    int sl = 1;
    while (sl * k < N) sl <<= 1;
    return sl;
}
}  // namespace

// padded states of a state row (0: more states than the kernel takes)
extern "C" int ttie_selective_state_pad(int N) { return N < 1 || N > 512 ? 0 : state_slices(N) * states_per_thread(N); }

// parts > 1: scratch holds requests * parts * channels * (padded states + 1) floats
extern "C" int ttie_selective_scan(const void* u, long long ld_u, const float* dt, long long ld_dt, const float* dt_bias, const float* A,
                                   const float* D, const void* bc, long long ld_bc, int col_b, int col_c, const void* z, long long ld_z,
                                   float* state, int state_rows, const void* xin, long long ld_x, float* tail, int tail_rows, int taps,
                                   const int* qsl, const int* slot_ids, int num_seqs, void* out, int I, int N, int parts, float* scratch,
                                   int dtype, void* stream) {
    if (num_seqs <= 0) return 0;
    if (N < 1 || N > 512) TTIE_FAIL("selective_scan: %d states per channel (1 to 512)", N);
    if (parts < 1 || (parts > 1 && !scratch) || (long long)num_seqs * parts > 65535)
        TTIE_FAIL("selective_scan: %d parts for %d requests", parts, num_seqs);
    if (taps > 1 && (!tail || !xin)) TTIE_FAIL("selective_scan: %d taps need state rows and inputs", taps);
    if (dtype != kF32 && dtype != kBF16) TTIE_FAIL("selective_scan: unknown dtype %d", dtype);
    SelArgs a;
    a.u = u; a.ld_u = ld_u; a.dt = dt; a.ld_dt = ld_dt; a.dt_bias = dt_bias; a.A = A; a.D = D; a.bc = bc; a.ld_bc = ld_bc; a.col_b = col_b;
    a.col_c = col_c; a.z = z; a.ld_z = ld_z; a.state = state; a.state_rows = state_rows; a.xin = xin; a.ld_x = ld_x; a.tail = tail;
    a.tail_rows = tail_rows; a.taps = taps; a.qsl = qsl; a.slot_ids = slot_ids; a.out = out; a.I = I; a.N = N;
    const int kpt = states_per_thread(N), sl = state_slices(N);
    a.Np = kpt * sl; a.parts = parts; a.scratch = scratch;
    a.scratch_dt = scratch ? scratch + (size_t)num_seqs * parts * I * a.Np : nullptr;
    const dim3 grid(ceil_div(I, NT / sl), num_seqs * parts);
    cudaStream_t s = (cudaStream_t)stream;
    for (int mode = parts > 1 ? 1 : 0; mode >= 0; --mode) {          // (mode 1: every part's own sum, from a zero state)
        a.mode = mode;
#define SEL_CASE(K, L_)                                                                                                   \
        if (kpt == K && sl == L_) {                                                                                       \
            if (dtype == kF32) TTIE_LAUNCH((selective_scan_kernel<float, K, L_>), grid, NT, 0, s, a);                     \
            else TTIE_LAUNCH((selective_scan_kernel<__nv_bfloat16, K, L_>), grid, NT, 0, s, a);                           \
        }
        SEL_CASE(4, 1) SEL_CASE(4, 2) SEL_CASE(4, 4) SEL_CASE(4, 8) SEL_CASE(4, 16) SEL_CASE(4, 32) SEL_CASE(8, 32) SEL_CASE(16, 32)
#undef SEL_CASE
        TTIE_CHECK_LAUNCH("selective_scan");
    }
    return 0;
}
