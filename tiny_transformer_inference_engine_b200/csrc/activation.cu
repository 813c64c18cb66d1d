// Elementwise functions between products, evaluated in 32-bit: out[i] = f(in[i]) for contiguous arrays, input and output
// each float32 or bfloat16 (in place when they are the same array).
//   0  relu(x)^2    1  tanh(x)    2  c * tanh(x / c) (a soft cap at +-c)    3  x    4  x * sigmoid(x) (silu)
// with x the input times `scale`.  activation_rows: the same on the first `cols` columns of rows with a stride, into contiguous
// 32-bit rows.
#include "common.cuh"
#include <math.h>
using namespace ttie;

namespace {

__device__ __forceinline__ float apply(float x, int kind, float c) {
    if (kind == 0) { const float r = fmaxf(x, 0.f); return r * r; }
    if (kind == 1) return tanhf(x);
    if (kind == 2) return c * tanhf(x / c);
    return kind == 4 ? x / (1.0f + expf(-x)) : x;
}

template <typename TI, typename TO>
__global__ void activation_kernel(const TI* __restrict__ in, TO* __restrict__ out, long long n, int kind, float c, float scale) {
    TTIE_PDL_ENTRY();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x)
        out[i] = from_f32<TO>(apply(to_f32(in[i]) * scale, kind, c));
}

// bfloat16 to bfloat16, eight values per thread (n a multiple of 8, both arrays 16-byte aligned)
__global__ void activation_bf16x8_kernel(const uint4* __restrict__ in, uint4* __restrict__ out, long long n8, int kind, float c, float scale) {
    TTIE_PDL_ENTRY();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n8; i += (long long)gridDim.x * blockDim.x) {
        const uint4 x = in[i];
        uint4 y;
        const __nv_bfloat162* a = reinterpret_cast<const __nv_bfloat162*>(&x);
        __nv_bfloat162* b = reinterpret_cast<__nv_bfloat162*>(&y);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 f = __bfloat1622float2(a[k]);
            b[k] = __floats2bfloat162_rn(apply(f.x * scale, kind, c), apply(f.y * scale, kind, c));
        }
        out[i] = y;
    }
}

template <typename T>
__global__ void activation_rows_kernel(const T* __restrict__ in, long long ld, float* __restrict__ out, int T_, int cols, int kind, float c,
                                       float scale) {
    TTIE_PDL_ENTRY();
    const int j = blockIdx.x * blockDim.x + threadIdx.x;             // grid: (columns, rows)
    if (j >= cols) return;
    for (size_t t = blockIdx.y; t < (size_t)T_; t += gridDim.y) out[t * cols + j] = apply(to_f32(in[t * ld + j]) * scale, kind, c);
}

// bfloat16 rows, eight values per thread (columns and row stride multiples of 8, 16-byte aligned arrays)
__global__ void activation_rows_vec8_kernel(const __nv_bfloat16* __restrict__ in, long long ld, float* __restrict__ out, int T_, int cols,
                                            int kind, float c, float scale) {
    TTIE_PDL_ENTRY();
    const int j = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
    if (j >= cols) return;
    for (size_t t = blockIdx.y; t < (size_t)T_; t += gridDim.y) {
        const uint4 x = *reinterpret_cast<const uint4*>(in + t * ld + j);
        const __nv_bfloat162* a = reinterpret_cast<const __nv_bfloat162*>(&x);
        float y[8];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 f = __bfloat1622float2(a[k]);
            y[2 * k] = apply(f.x * scale, kind, c); y[2 * k + 1] = apply(f.y * scale, kind, c);
        }
        float4* o = reinterpret_cast<float4*>(out + t * cols + j);
        o[0] = make_float4(y[0], y[1], y[2], y[3]);
        o[1] = make_float4(y[4], y[5], y[6], y[7]);
    }
}

}  // namespace

// out[i] = sum over s of part[s * stride + i], added in order
template <typename T>
__global__ void sum_partials_kernel(const float* __restrict__ part, int S, long long stride, T* __restrict__ out, long long n) {
    TTIE_PDL_ENTRY();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    float acc = 0.f;
#pragma unroll 4
    for (int s = 0; s < S; ++s) acc += part[s * stride + i];
    out[i] = from_f32<T>(acc);
}

extern "C" int ttie_sum_partials(const float* part, int S, long long stride, void* out, long long n, int dtype, void* stream) {
    if (n <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    const unsigned blocks = (unsigned)((n + 127) / 128);
    if (dtype == kF32) TTIE_LAUNCH(sum_partials_kernel<float>, blocks, 128, 0, s, part, S, stride, (float*)out, n);
    else if (dtype == kBF16) TTIE_LAUNCH(sum_partials_kernel<__nv_bfloat16>, blocks, 128, 0, s, part, S, stride, (__nv_bfloat16*)out, n);
    else TTIE_FAIL("sum_partials: unknown dtype %d", dtype);
    TTIE_CHECK_LAUNCH("sum_partials");
    return 0;
}

extern "C" int ttie_activation_rows(const void* in, long long ld, float* out, int T, int cols, int kind, float c, float scale, int dtype, void* stream) {
    if (T <= 0 || cols <= 0) return 0;
    if (kind < 0 || kind > 4) TTIE_FAIL("activation_rows: unknown kind %d", kind);
    if (kind == 2 && !(c > 0.f)) TTIE_FAIL("activation_rows: a soft cap needs a positive constant");
    cudaStream_t s = (cudaStream_t)stream;
    const int rows = T < 65535 ? T : 65535;
    if (dtype == kBF16 && cols % 8 == 0 && ld % 8 == 0 && !(((uintptr_t)in | (uintptr_t)out) & 15))
        TTIE_LAUNCH(activation_rows_vec8_kernel, dim3(ceil_div(cols / 8, 128), rows), 128, 0, s, (const __nv_bfloat16*)in, ld, out, T, cols, kind, c, scale);
    else if (dtype == kBF16) TTIE_LAUNCH(activation_rows_kernel<__nv_bfloat16>, dim3(ceil_div(cols, 256), rows), 256, 0, s, (const __nv_bfloat16*)in, ld, out, T, cols, kind, c, scale);
    else if (dtype == kF32) TTIE_LAUNCH(activation_rows_kernel<float>, dim3(ceil_div(cols, 256), rows), 256, 0, s, (const float*)in, ld, out, T, cols, kind, c, scale);
    else TTIE_FAIL("activation_rows: unknown dtype %d", dtype);
    TTIE_CHECK_LAUNCH("activation_rows");
    return 0;
}

extern "C" int ttie_activation(const void* in, void* out, long long n, int kind, float c, float scale, int in_dtype, int out_dtype, void* stream) {
    if (n <= 0) return 0;
    if (kind < 0 || kind > 4) TTIE_FAIL("activation: unknown kind %d", kind);
    if (kind == 2 && !(c > 0.f)) TTIE_FAIL("activation: a soft cap needs a positive constant");
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = 256;
    if (in_dtype == kBF16 && out_dtype == kBF16 && n % 8 == 0 && !(((uintptr_t)in | (uintptr_t)out) & 15)) {
        const long long n8 = n / 8;
        const int grid = (int)((n8 + threads - 1) / threads < 148LL * 16 ? (n8 + threads - 1) / threads : 148LL * 16);
        TTIE_LAUNCH(activation_bf16x8_kernel, grid, threads, 0, s, (const uint4*)in, (uint4*)out, n8, kind, c, scale);
        TTIE_CHECK_LAUNCH("activation");
        return 0;
    }
    const int grid = (int)((n + threads - 1) / threads < 148LL * 32 ? (n + threads - 1) / threads : 148LL * 32);
    if (in_dtype == kF32 && out_dtype == kF32) TTIE_LAUNCH((activation_kernel<float, float>), grid, threads, 0, s, (const float*)in, (float*)out, n, kind, c, scale);
    else if (in_dtype == kF32 && out_dtype == kBF16) TTIE_LAUNCH((activation_kernel<float, __nv_bfloat16>), grid, threads, 0, s, (const float*)in, (__nv_bfloat16*)out, n, kind, c, scale);
    else if (in_dtype == kBF16 && out_dtype == kBF16) TTIE_LAUNCH((activation_kernel<__nv_bfloat16, __nv_bfloat16>), grid, threads, 0, s, (const __nv_bfloat16*)in, (__nv_bfloat16*)out, n, kind, c, scale);
    else if (in_dtype == kBF16 && out_dtype == kF32) TTIE_LAUNCH((activation_kernel<__nv_bfloat16, float>), grid, threads, 0, s, (const __nv_bfloat16*)in, (float*)out, n, kind, c, scale);
    else TTIE_FAIL("activation: unknown dtypes %d -> %d", in_dtype, out_dtype);
    TTIE_CHECK_LAUNCH("activation");
    return 0;
}
