// The norm step of layers that norm a sub-layer's output before it is added (and the next sub-layer's input as ever):
//     x <- x + delta / sqrt(mean(delta^2) + eps_b) * w_b          out = x / sqrt(mean(x^2) + eps) * w
// x is the 32-bit residual stream, rewritten in place; delta the sub-layer's output, [R, d] in the compute dtype or 32-bit
// partial sums [S, R, d] of a K-split product (added in the order s = 0 .. S-1).  One pass over the row: it stays in registers
// (or shared memory) between the two reductions.  With a row list the rows are gathered into `out` and the stream is left alone.
//   sandwich_cluster_kernel   few rows of a wide model (decode steps): a cluster of C CTAs shares a row, each reduces its share and
//                             the shares are added in rank order through distributed shared memory
//   sandwich_vec_kernel       one CTA per row, four values per load
//   sandwich_kernel           any width, the row in shared memory
#include "common.cuh"
using namespace ttie;

namespace {

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const __nv_bfloat16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
    uint2 o;
    *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(v.x, v.y);
    *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = o;
}
__device__ __forceinline__ float sq4(float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }
__device__ __forceinline__ float4 axpy4(float4 y, float f, float4 w, float4 x) {       // x + y * f * w
    return make_float4(x.x + y.x * f * w.x, x.y + y.y * f * w.y, x.z + y.z * f * w.z, x.w + y.w * f * w.w);
}

template <typename T> struct SandwichArgs {
    float* resid; const T* delta; const float* dpart; int S; long long part_stride; const int* rows;
    const float* wb; const float* w; T* out; int d; float eps_b, eps;
};

template <typename T>
__device__ __forceinline__ float4 load_delta4(const SandwichArgs<T>& a, size_t at) {
    if (a.delta) return ld4(a.delta + at);
    float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s0 = 0; s0 < a.S; s0 += 4) {                            // four loads in flight, added in order
        float4 b[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) if (s0 + k < a.S) b[k] = ld4(a.dpart + (s0 + k) * a.part_stride + at);
#pragma unroll
        for (int k = 0; k < 4; ++k) if (s0 + k < a.S) { t.x += b[k].x; t.y += b[k].y; t.z += b[k].z; t.w += b[k].w; }
    }
    return t;
}

template <typename T, int NT, int MAXC>
__global__ void __launch_bounds__(NT) sandwich_vec_kernel(const SandwichArgs<T> a) {
    __shared__ float scratch[32];
    TTIE_PDL_ENTRY();
    const int r = blockIdx.x, nchunk = a.d >> 2;
    const size_t src = (size_t)(a.rows ? a.rows[r] : r) * a.d;
    float4 y[MAXC], x[MAXC];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < MAXC; ++c) {
        const int ch = threadIdx.x + c * NT;
        if (ch < nchunk) { x[c] = ld4(a.resid + src + ch * 4); y[c] = load_delta4(a, src + ch * 4); ss += sq4(y[c]); }
    }
    ss = block_sum(ss, scratch);
    const float inv_b = 1.0f / sqrtf(ss / (float)a.d + a.eps_b);
    ss = 0.f;
#pragma unroll
    for (int c = 0; c < MAXC; ++c) {
        const int ch = threadIdx.x + c * NT;
        if (ch < nchunk) {
            x[c] = axpy4(y[c], inv_b, ld4(a.wb + ch * 4), x[c]);
            if (!a.rows) st4(a.resid + src + ch * 4, x[c]);
            ss += sq4(x[c]);
        }
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)a.d + a.eps);
#pragma unroll
    for (int c = 0; c < MAXC; ++c) {
        const int ch = threadIdx.x + c * NT;
        if (ch < nchunk) st4(a.out + (size_t)r * a.d + ch * 4, axpy4(x[c], inv, ld4(a.w + ch * 4), make_float4(0.f, 0.f, 0.f, 0.f)));
    }
}

// sum over the CTAs of a cluster of one float each, in rank order
template <int C>
__device__ __forceinline__ float cluster_total(const float* share) {
    asm volatile("barrier.cluster.arrive.release.aligned;\nbarrier.cluster.wait.acquire.aligned;" ::: "memory");
    float total = 0.f;
#pragma unroll
    for (int k = 0; k < C; ++k) {
        uint32_t remote;
        float part;
        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"((uint32_t)__cvta_generic_to_shared(share)), "r"(k));
        asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(part) : "r"(remote) : "memory");
        total += part;
    }
    return total;
}

template <typename T, int NT, int MAXC, int C>
__global__ void __launch_bounds__(NT) sandwich_cluster_kernel(const SandwichArgs<T> a) {
    __shared__ float scratch[32];
    __shared__ float share[2];                                       // this CTA's part of either sum of squares
    const int r = blockIdx.x / C, rank = blockIdx.x - r * C;         // clusters are consecutive CTAs along x
    const int nchunk = a.d >> 2, per = (nchunk + C - 1) / C;
    const int c0 = rank * per, c1 = min(nchunk, c0 + per);
    float4 wb[MAXC], w[MAXC];
#pragma unroll
    for (int c = 0; c < MAXC; ++c) {                                 // (weights do not depend on the kernel before this one)
        const int ch = c0 + threadIdx.x + c * NT;
        if (ch < c1) { wb[c] = ld4(a.wb + ch * 4); w[c] = ld4(a.w + ch * 4); }
    }
    TTIE_PDL_ENTRY();
    const size_t src = (size_t)(a.rows ? a.rows[r] : r) * a.d;
    float4 y[MAXC], x[MAXC];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < MAXC; ++c) {
        const int ch = c0 + threadIdx.x + c * NT;
        if (ch < c1) { x[c] = ld4(a.resid + src + ch * 4); y[c] = load_delta4(a, src + ch * 4); ss += sq4(y[c]); }
    }
    ss = block_sum(ss, scratch);
    if (threadIdx.x == 0) share[0] = ss;
    const float inv_b = 1.0f / sqrtf(cluster_total<C>(&share[0]) / (float)a.d + a.eps_b);
    ss = 0.f;
#pragma unroll
    for (int c = 0; c < MAXC; ++c) {
        const int ch = c0 + threadIdx.x + c * NT;
        if (ch < c1) {
            x[c] = axpy4(y[c], inv_b, wb[c], x[c]);
            if (!a.rows) st4(a.resid + src + ch * 4, x[c]);
            ss += sq4(x[c]);
        }
    }
    ss = block_sum(ss, scratch);
    if (threadIdx.x == 0) share[1] = ss;
    const float inv = 1.0f / sqrtf(cluster_total<C>(&share[1]) / (float)a.d + a.eps);
#pragma unroll
    for (int c = 0; c < MAXC; ++c) {
        const int ch = c0 + threadIdx.x + c * NT;
        if (ch < c1) st4(a.out + (size_t)r * a.d + ch * 4, axpy4(x[c], inv, w[c], make_float4(0.f, 0.f, 0.f, 0.f)));
    }
    // no CTA may leave while another still reads its shares
    asm volatile("barrier.cluster.arrive.release.aligned;\nbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}

template <typename T>
__global__ void __launch_bounds__(256) sandwich_kernel(const SandwichArgs<T> a) {
    extern __shared__ float row[];
    __shared__ float scratch[32];
    TTIE_PDL_ENTRY();
    const int r = blockIdx.x;
    const size_t src = (size_t)(a.rows ? a.rows[r] : r) * a.d;
    float ss = 0.f;
    for (int i = threadIdx.x; i < a.d; i += blockDim.x) {
        float v = a.delta ? to_f32(a.delta[src + i]) : 0.f;
        if (!a.delta) for (int s = 0; s < a.S; ++s) v += a.dpart[(size_t)s * a.part_stride + src + i];
        row[i] = v;
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float inv_b = 1.0f / sqrtf(ss / (float)a.d + a.eps_b);
    ss = 0.f;
    for (int i = threadIdx.x; i < a.d; i += blockDim.x) {
        const float v = a.resid[src + i] + row[i] * inv_b * a.wb[i];
        row[i] = v;
        if (!a.rows) a.resid[src + i] = v;
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)a.d + a.eps);
    for (int i = threadIdx.x; i < a.d; i += blockDim.x) a.out[(size_t)r * a.d + i] = from_f32<T>(row[i] * inv * a.w[i]);
}

template <typename T>
int launch(const SandwichArgs<T>& a, int R, cudaStream_t s) {
    const bool aligned = !(((uintptr_t)a.resid | (uintptr_t)a.delta | (uintptr_t)a.dpart | (uintptr_t)a.wb | (uintptr_t)a.w | (uintptr_t)a.out) & 15)
                         && a.part_stride % 4 == 0;
    if (a.d % 4 == 0 && aligned && a.d >= 1024 && a.d <= 8192 && R <= 96)
        TTIE_LAUNCH_CLUSTER((sandwich_cluster_kernel<T, 256, 2, 4>), R * 4, 256, 0, s, 4, a);
    else if (a.d % 4 == 0 && aligned && a.d <= 2048) TTIE_LAUNCH((sandwich_vec_kernel<T, 128, 4>), R, 128, 0, s, a);
    else if (a.d % 4 == 0 && aligned && a.d <= 8192) TTIE_LAUNCH((sandwich_vec_kernel<T, 256, 8>), R, 256, 0, s, a);
    else {
        const size_t smem = (size_t)a.d * sizeof(float);
        if (smem > 200 * 1024) TTIE_FAIL("sandwich_norm: width %d needs %zu bytes of shared memory (limit 204800)", a.d, smem);
        if (smem > 48 * 1024) cudaFuncSetAttribute(sandwich_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        TTIE_LAUNCH(sandwich_kernel<T>, R, 256, smem, s, a);
    }
    TTIE_CHECK_LAUNCH("sandwich_norm");
    return 0;
}
}  // namespace

// delta: [rows of resid, d] in the compute dtype, or null and dpart: 32-bit partial sums [S][rows of resid][d].  Weights are 32-bit.
extern "C" int ttie_sandwich_norm(float* resid, const void* delta, const float* dpart, int S, long long part_stride, const int* rows,
                                  const float* wb, float eps_b, const float* w, float eps, void* out, int R, int d, int dtype, void* stream) {
    if (R <= 0) return 0;
    if (!delta && (!dpart || S < 1)) TTIE_FAIL("sandwich_norm: no sub-layer output");
    if (dtype == kF32) return launch<float>({resid, (const float*)delta, dpart, S, part_stride, rows, wb, w, (float*)out, d, eps_b, eps}, R, (cudaStream_t)stream);
    if (dtype == kBF16) return launch<__nv_bfloat16>({resid, (const __nv_bfloat16*)delta, dpart, S, part_stride, rows, wb, w, (__nv_bfloat16*)out, d, eps_b, eps}, R, (cudaStream_t)stream);
    TTIE_FAIL("sandwich_norm: unknown dtype %d", dtype);
}
