// Kernels of layers whose sub-layers all read the same normed rows and are added to the stream in one go, and of the input that a
// token's id gives every layer.
//   residual_sum   x <- x + mult * (a + f + bias): x the 32-bit stream, rewritten in place; a and f sub-layers' outputs, each [T, d] in
//                  the compute dtype or 32-bit partial sums [S, T, d] of a K-split product (added in the order s = 0 .. S-1); f may
//                  instead be rows of routed experts that all weigh the same, weight * sum_k Y[pos(t, k), :] in the order of k;
//                  bias 32-bit [d].  Optionally the new rows also leave in the compute dtype (for a sub-layer that reads the stream).
//   token_gate     g[t, j] = gelu_tanh(z[t, j]) * E[id_t, col0 + j]: z a gate's product [T, N] in the compute dtype or 32-bit partial sums
//                  [S, T, N]; E [vocab, ld] a table with a row per token id, of which one layer takes the columns col0 .. col0 + n.
//                  N >= n: the columns from n on are padding and leave as zeros.
#include "common.cuh"
using namespace ttie;

namespace {

struct Term { const void* rows; const float* part; int S; long long stride; };
struct ExpertRows { const void* y; const int* pos; int top; float weight; };

template <int V> struct Vals { float v[V]; };
// V values at p: V 1, or a multiple of 4 at a place aligned to four (32-bit) or V (16-bit) values
template <int V> __device__ __forceinline__ Vals<V> ldv(const float* p) {
    Vals<V> r;
    if (V == 1) r.v[0] = p[0];
    else {
#pragma unroll
        for (int i = 0; i < V; i += 4) {
            const float4 x = *reinterpret_cast<const float4*>(p + i);
            r.v[i] = x.x; r.v[(i + 1) % V] = x.y; r.v[(i + 2) % V] = x.z; r.v[(i + 3) % V] = x.w;
        }
    }
    return r;
}
template <int V> __device__ __forceinline__ Vals<V> ldv(const __nv_bfloat16* p) {
    Vals<V> r;
    if (V == 1) r.v[0] = __bfloat162float(p[0]);
    else {
        __align__(16) __nv_bfloat162 h[(V + 1) / 2];
        if (V == 8) *reinterpret_cast<uint4*>(h) = *reinterpret_cast<const uint4*>(p);
        else *reinterpret_cast<uint2*>(h) = *reinterpret_cast<const uint2*>(p);
#pragma unroll
        for (int i = 0; i < V / 2; ++i) { const float2 f = __bfloat1622float2(h[i]); r.v[2 * i] = f.x; r.v[(2 * i + 1) % V] = f.y; }
    }
    return r;
}
template <int V> __device__ __forceinline__ void stv(float* p, const Vals<V>& r) {
    if (V == 1) p[0] = r.v[0];
    else {
#pragma unroll
        for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(r.v[i], r.v[(i + 1) % V], r.v[(i + 2) % V], r.v[(i + 3) % V]);
    }
}
template <int V> __device__ __forceinline__ void stv(__nv_bfloat16* p, const Vals<V>& r) {
    if (V == 1) p[0] = __float2bfloat16_rn(r.v[0]);
    else {
        __align__(16) __nv_bfloat162 h[(V + 1) / 2];
#pragma unroll
        for (int i = 0; i < V / 2; ++i) h[i] = __floats2bfloat162_rn(r.v[2 * i], r.v[(2 * i + 1) % V]);
        if (V == 8) *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(h);
        else *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(h);
    }
}
template <int V> __device__ __forceinline__ void addv(Vals<V>& a, const Vals<V>& b) {
#pragma unroll
    for (int i = 0; i < V; ++i) a.v[i] += b.v[i];
}
// the partial sums of a product at one place: a few loads in flight, added in order
template <int V> __device__ __forceinline__ Vals<V> sum_parts(const float* part, int S, long long stride) {
    constexpr int AT_ONCE = V == 8 ? 2 : 4;
    Vals<V> t;
#pragma unroll
    for (int i = 0; i < V; ++i) t.v[i] = 0.f;
    for (int s0 = 0; s0 < S; s0 += AT_ONCE) {
        Vals<V> b[AT_ONCE];
#pragma unroll
        for (int k = 0; k < AT_ONCE; ++k) if (s0 + k < S) b[k] = ldv<V>(part + (s0 + k) * stride);
#pragma unroll
        for (int k = 0; k < AT_ONCE; ++k) if (s0 + k < S) addv<V>(t, b[k]);
    }
    return t;
}
template <typename T, int V> __device__ __forceinline__ void add_term(Vals<V>& sum, const Term& m, size_t at) {
    if (m.rows) addv<V>(sum, ldv<V>(reinterpret_cast<const T*>(m.rows) + at));
    else if (m.part) addv<V>(sum, sum_parts<V>(m.part + at, m.S, m.stride));
}

template <typename T, typename TY, int V>
__global__ void __launch_bounds__(128) residual_sum_kernel(float* __restrict__ x, const Term a, const Term f, const ExpertRows ex,
                                                           const float* __restrict__ bias, float mult, T* __restrict__ out, int T_, int d) {
    TTIE_PDL_ENTRY();
    const int i = (blockIdx.x * blockDim.x + threadIdx.x) * V;      // grid: (columns, rows)
    if (i >= d) return;
    for (size_t t = blockIdx.y; t < (size_t)T_; t += gridDim.y) {
        const size_t at = t * d + i;
        Vals<V> xv = ldv<V>(x + at), sum;
#pragma unroll
        for (int k = 0; k < V; ++k) sum.v[k] = 0.f;
        add_term<T, V>(sum, a, at);
        add_term<T, V>(sum, f, at);
        if (ex.y) {
            Vals<V> e;
#pragma unroll
            for (int k = 0; k < V; ++k) e.v[k] = 0.f;
            constexpr int AT_ONCE = V == 8 ? 2 : 4;
            for (int k0 = 0; k0 < ex.top; k0 += AT_ONCE) {           // a few rows in flight, added in order
                Vals<V> b[AT_ONCE];
#pragma unroll
                for (int k = 0; k < AT_ONCE; ++k)
                    if (k0 + k < ex.top) b[k] = ldv<V>(reinterpret_cast<const TY*>(ex.y) + (size_t)ex.pos[t * ex.top + k0 + k] * d + i);
#pragma unroll
                for (int k = 0; k < AT_ONCE; ++k) if (k0 + k < ex.top) addv<V>(e, b[k]);
            }
#pragma unroll
            for (int k = 0; k < V; ++k) sum.v[k] = fmaf(ex.weight, e.v[k], sum.v[k]);
        }
        if (bias) addv<V>(sum, ldv<V>(bias + i));
#pragma unroll
        for (int k = 0; k < V; ++k) xv.v[k] = fmaf(mult, sum.v[k], xv.v[k]);
        stv<V>(x + at, xv);
        if (out) stv<V>(out + at, xv);
    }
}

template <typename T, int V>
__global__ void __launch_bounds__(128) token_gate_kernel(const T* __restrict__ z, const float* __restrict__ part, int S, long long stride,
                                                         const int* __restrict__ ids, const T* __restrict__ table, long long ld, int vocab,
                                                         int col0, int n, int N, unsigned total, T* __restrict__ out) {
    TTIE_PDL_ENTRY();
    const unsigned per = (unsigned)N / V;                            // groups of V columns of a row
    for (unsigned e = blockIdx.x * blockDim.x + threadIdx.x; e < total; e += gridDim.x * blockDim.x) {
        const unsigned t = e / per;
        const int j = (int)(e - t * per) * V;
        const size_t at = (size_t)t * N + j;
        const int id = min(max(ids[t], 0), vocab - 1);              // ids are validated on the host; never read outside
        const T* row = table + (size_t)id * ld + col0 + j;
        Vals<V> g, r;
        if (V > 1) r = ldv<V>(row);                                  // (the whole group lies inside: n is a multiple of V)
        else r.v[0] = j < n ? to_f32(row[0]) : 0.f;
        g = z ? ldv<V>(z + at) : sum_parts<V>(part + at, S, stride);
#pragma unroll
        for (int i = 0; i < V; ++i) g.v[i] = V > 1 || j < n ? gelu_tanh(g.v[i]) * r.v[i] : 0.f;
        stv<V>(out + at, g);
    }
}

template <typename T, typename TY>
int launch_sum(float* x, const Term& a, const Term& f, const ExpertRows& ex, const float* bias, float mult, void* out, int T_, int d, cudaStream_t s) {
    const bool aligned = a.stride % 4 == 0 && f.stride % 4 == 0
                         && !(((uintptr_t)x | (uintptr_t)a.rows | (uintptr_t)a.part | (uintptr_t)f.rows | (uintptr_t)f.part | (uintptr_t)ex.y | (uintptr_t)bias | (uintptr_t)out) & 15);
    // prompt portions: eight values per thread (16-byte loads of the 16-bit rows); a few rows: four, so that more threads share them
    const int V = aligned && d % 8 == 0 && sizeof(T) == 2 && (long long)T_ * d >= (1 << 20) ? 8 : aligned && d % 4 == 0 ? 4 : 1;
    const dim3 grid(ceil_div(d / V, 128), T_ < 65535 ? T_ : 65535);
    if (V == 8) TTIE_LAUNCH((residual_sum_kernel<T, TY, 8>), grid, 128, 0, s, x, a, f, ex, bias, mult, (T*)out, T_, d);
    else if (V == 4) TTIE_LAUNCH((residual_sum_kernel<T, TY, 4>), grid, 128, 0, s, x, a, f, ex, bias, mult, (T*)out, T_, d);
    else TTIE_LAUNCH((residual_sum_kernel<T, TY, 1>), grid, 128, 0, s, x, a, f, ex, bias, mult, (T*)out, T_, d);
    TTIE_CHECK_LAUNCH("residual_sum");
    return 0;
}

template <typename T>
int launch_gate(const void* z, const float* part, int S, long long stride, const int* ids, const void* table, long long ld, int vocab, int col0,
                int n, int N, int T_, void* out, cudaStream_t s) {
    constexpr int VW = 4;
    const bool vec = n == N && n % VW == 0 && col0 % VW == 0 && ld % VW == 0 && stride % VW == 0
                     && !(((uintptr_t)z | (uintptr_t)part | (uintptr_t)table | (uintptr_t)out) & 15);
    const long long total = (long long)T_ * N / (vec ? VW : 1);
    if (total >= (1LL << 31)) TTIE_FAIL("token_gate: %d rows of %d values in one launch", T_, N);
    const int grid = (int)((total + 127) / 128 < 8192 ? (total + 127) / 128 : 8192);
    if (vec) TTIE_LAUNCH((token_gate_kernel<T, VW>), grid, 128, 0, s, (const T*)z, part, S, stride, ids, (const T*)table, ld, vocab, col0, n, N, (unsigned)total, (T*)out);
    else TTIE_LAUNCH((token_gate_kernel<T, 1>), grid, 128, 0, s, (const T*)z, part, S, stride, ids, (const T*)table, ld, vocab, col0, n, N, (unsigned)total, (T*)out);
    TTIE_CHECK_LAUNCH("token_gate");
    return 0;
}
}  // namespace

// a / f: rows [T, d] in the compute dtype, or null and partial sums [S][T][d], or both null (no such term); y: expert rows of dtype
// y_dtype with pos int32 [T][top], or null; out: [T, d] in the compute dtype, or null
extern "C" int ttie_residual_sum(float* x, const void* a_rows, const float* a_part, int a_S, long long a_stride, const void* f_rows,
                                 const float* f_part, int f_S, long long f_stride, const void* y, int y_dtype, const int* pos, int top,
                                 float weight, const float* bias, float mult, void* out, int T, int d, int dtype, void* stream) {
    if (T <= 0 || d <= 0) return 0;
    if (y && (!pos || top < 1)) TTIE_FAIL("residual_sum: expert rows need their places");
    const Term a{a_rows, a_part, a_S, a_stride}, f{f_rows, f_part, f_S, f_stride};
    const ExpertRows ex{y, pos, top, weight};
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == kF32 && (!y || y_dtype == kF32)) return launch_sum<float, float>(x, a, f, ex, bias, mult, out, T, d, s);
    if (dtype == kBF16 && y && y_dtype == kBF16) return launch_sum<__nv_bfloat16, __nv_bfloat16>(x, a, f, ex, bias, mult, out, T, d, s);
    if (dtype == kBF16) return launch_sum<__nv_bfloat16, float>(x, a, f, ex, bias, mult, out, T, d, s);
    TTIE_FAIL("residual_sum: dtype %d with expert rows of dtype %d", dtype, y_dtype);
}

extern "C" int ttie_token_gate(const void* z, const float* part, int S, long long stride, const int* ids, const void* table, long long ld,
                               int vocab, int col0, int n, int N, int T, void* out, int dtype, void* stream) {
    if (T <= 0 || N <= 0) return 0;
    if (!z && (!part || S < 1)) TTIE_FAIL("token_gate: no gate values");
    if (col0 < 0 || n < 1 || n > N || col0 + n > ld) TTIE_FAIL("token_gate: columns %d .. %d of a table of %lld, %d gate values", col0, col0 + n, ld, N);
    if (dtype == kF32) return launch_gate<float>(z, part, S, stride, ids, table, ld, vocab, col0, n, N, T, out, (cudaStream_t)stream);
    if (dtype == kBF16) return launch_gate<__nv_bfloat16>(z, part, S, stride, ids, table, ld, vocab, col0, n, N, T, out, (cudaStream_t)stream);
    TTIE_FAIL("token_gate: unknown dtype %d", dtype);
}
