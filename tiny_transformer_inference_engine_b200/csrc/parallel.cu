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
template <int V> __device__ __forceinline__ Vals<V> ldv(const float* p) {
    Vals<V> r;
    if (V == 4) { const float4 x = *reinterpret_cast<const float4*>(p); r.v[0] = x.x; r.v[1 % V] = x.y; r.v[2 % V] = x.z; r.v[3 % V] = x.w; }
    else r.v[0] = p[0];
    return r;
}
template <int V> __device__ __forceinline__ Vals<V> ldv(const __nv_bfloat16* p) {
    Vals<V> r;
    if (V == 4) {
        const uint2 x = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.y));
        r.v[0] = a.x; r.v[1 % V] = a.y; r.v[2 % V] = b.x; r.v[3 % V] = b.y;
    } else r.v[0] = __bfloat162float(p[0]);
    return r;
}
template <int V> __device__ __forceinline__ void stv(float* p, const Vals<V>& r) {
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1 % V], r.v[2 % V], r.v[3 % V]);
    else p[0] = r.v[0];
}
template <int V> __device__ __forceinline__ void stv(__nv_bfloat16* p, const Vals<V>& r) {
    if (V == 4) {
        uint2 o;
        *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(r.v[0], r.v[1 % V]);
        *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(r.v[2 % V], r.v[3 % V]);
        *reinterpret_cast<uint2*>(p) = o;
    } else p[0] = __float2bfloat16_rn(r.v[0]);
}
template <int V> __device__ __forceinline__ void addv(Vals<V>& a, const Vals<V>& b) {
#pragma unroll
    for (int i = 0; i < V; ++i) a.v[i] += b.v[i];
}
// the partial sums of a product at one place: four loads in flight, added in order
template <int V> __device__ __forceinline__ Vals<V> sum_parts(const float* part, int S, long long stride) {
    Vals<V> t;
#pragma unroll
    for (int i = 0; i < V; ++i) t.v[i] = 0.f;
    for (int s0 = 0; s0 < S; s0 += 4) {
        Vals<V> b[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) if (s0 + k < S) b[k] = ldv<V>(part + (s0 + k) * stride);
#pragma unroll
        for (int k = 0; k < 4; ++k) if (s0 + k < S) addv<V>(t, b[k]);
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
            for (int k0 = 0; k0 < ex.top; k0 += 4) {                 // four rows in flight, added in order
                Vals<V> b[4];
#pragma unroll
                for (int k = 0; k < 4; ++k)
                    if (k0 + k < ex.top) b[k] = ldv<V>(reinterpret_cast<const TY*>(ex.y) + (size_t)ex.pos[t * ex.top + k0 + k] * d + i);
#pragma unroll
                for (int k = 0; k < 4; ++k) if (k0 + k < ex.top) addv<V>(e, b[k]);
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

template <typename T>
__global__ void __launch_bounds__(128) token_gate_kernel(const T* __restrict__ z, const float* __restrict__ part, int S, long long stride,
                                                         const int* __restrict__ ids, const T* __restrict__ table, long long ld, int vocab,
                                                         int col0, int n, int N, long long total, T* __restrict__ out) {
    TTIE_PDL_ENTRY();
    for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
        const long long t = e / N;
        const int j = (int)(e - t * N);
        float g = 0.f;
        if (j < n) {
            const int id = min(max(ids[t], 0), vocab - 1);          // ids are validated on the host; never read outside
            const float v = z ? to_f32(z[e]) : sum_parts<1>(part + e, S, stride).v[0];
            g = gelu_tanh(v) * to_f32(table[(size_t)id * ld + col0 + j]);
        }
        out[e] = from_f32<T>(g);
    }
}

template <typename T, typename TY>
int launch_sum(float* x, const Term& a, const Term& f, const ExpertRows& ex, const float* bias, float mult, void* out, int T_, int d, cudaStream_t s) {
    const bool vec = d % 4 == 0 && a.stride % 4 == 0 && f.stride % 4 == 0
                     && !(((uintptr_t)x | (uintptr_t)a.rows | (uintptr_t)a.part | (uintptr_t)f.rows | (uintptr_t)f.part | (uintptr_t)ex.y | (uintptr_t)bias | (uintptr_t)out) & 15);
    const dim3 grid(ceil_div(vec ? d / 4 : d, 128), T_ < 65535 ? T_ : 65535);
    if (vec) TTIE_LAUNCH((residual_sum_kernel<T, TY, 4>), grid, 128, 0, s, x, a, f, ex, bias, mult, (T*)out, T_, d);
    else TTIE_LAUNCH((residual_sum_kernel<T, TY, 1>), grid, 128, 0, s, x, a, f, ex, bias, mult, (T*)out, T_, d);
    TTIE_CHECK_LAUNCH("residual_sum");
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
    const long long total = (long long)T * N;
    const int grid = (int)((total + 127) / 128 < 8192 ? (total + 127) / 128 : 8192);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == kF32) TTIE_LAUNCH(token_gate_kernel<float>, grid, 128, 0, s, (const float*)z, part, S, stride, ids, (const float*)table, ld, vocab, col0, n, N, total, (float*)out);
    else if (dtype == kBF16) TTIE_LAUNCH(token_gate_kernel<__nv_bfloat16>, grid, 128, 0, s, (const __nv_bfloat16*)z, part, S, stride, ids, (const __nv_bfloat16*)table, ld, vocab, col0, n, N, total, (__nv_bfloat16*)out);
    else TTIE_FAIL("token_gate: unknown dtype %d", dtype);
    TTIE_CHECK_LAUNCH("token_gate");
    return 0;
}
