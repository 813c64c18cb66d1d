// Attention whose score rows are mixed over the heads before the softmax ("talking heads"): head h attends with
//     score_h(i, j) = sum_g M[h, g] (q_g(i) . k_kv(g)(j)) * scale.
// The sum is linear in the queries, so it need not be formed per key.  With the keys of all kv heads of a token laid side by
// side as one row K_j (G heads of D values), score_h is the product of K_j with ONE mixed query row per head,
//     Q_h(i) = [ sum over g of kv head c of M[h, g] q_g(i) ]  for c = 0 .. G-1,
// and every attention kernel of the package computes it as H query heads on one shared key head of G * D values.
//
//   joint_qkv_store   one CTA per (token, run of output heads).  The token's projected row [q | k | v] is read once: one root mean square
//                     over all of q and one over all of k (with weights per channel; optional), the rotation of the first
//                     `rot` values of every head, the mixing in 32-bit and the write of Q as [T, H, W] (W >= G * D, the rest
//                     zero); keys and values go into the pages as joint rows [page, slot, W], values optionally blended with
//                     those of an earlier layer, (1 - mix) * v + mix * v_first.
//   joint_values      drops what a joint value row holds of the other kv heads: out[t, h] = attn[t, h, kv(h) * Dv ..].
#include "common.cuh"
using namespace ttie;

namespace {

struct JointStoreArgs {
    const void* proj; long long ld;                                  // [T, >= H*D + G*D + G*Dv]
    int H, G, D, Dv, W;
    const float* mix;                                                // [H, H] transposed: mix[g * H + h] is the weight of head g's scores in head h's
    const float* norm_w; float eps;                                  // [H*D + G*D] or null
    const float2* cs; int rot, style;
    const void* v_first; long long ld_first; float v_mix;            // [T, G*Dv] (a view with a row stride) or null
    const int* positions; const int* token_seq;
    const int* block_table; int table_width, page_size, num_pages, write_kv;
    void* q_out; void* k_pages; void* v_pages;
    int heads_per_cta;
};

constexpr int MIXT = 256, HB = 8;           // threads; output heads a thread carries at a time

// sums of squares of two ranges at once: (over q, over k)
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* scratch) {
    a = warp_sum(a); b = warp_sum(b);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    __syncthreads();
    if (lane == 0) scratch[warp] = make_float2(a, b);
    __syncthreads();
    float2 t = make_float2(0.f, 0.f);
#pragma unroll
    for (int w = 0; w < MIXT / 32; ++w) { t.x += scratch[w].x; t.y += scratch[w].y; }      // (fixed order, the same for every thread)
    return t;
}

// rotates the first `rot` values of `heads` rows of D values in place (pairs are disjoint: no two threads share one)
__device__ __forceinline__ void rotate_rows(float* x, int heads, int D, int rot, int style, const float2* cs) {
    const int half = rot >> 1;
    for (int e = threadIdx.x; e < heads * half; e += blockDim.x) {
        const int h = e / half, i = e - h * half;
        float* a = x + h * D + (style == 1 ? i : 2 * i);
        float* b = style == 1 ? a + half : a + 1;
        const float2 c = cs[i];
        const float u = *a, v = *b;
        *a = u * c.x - v * c.y;
        *b = v * c.x + u * c.y;
    }
}

// (d0, d1) += (a0, a1) * b, one instruction (fma.rn.f32x2)
__device__ __forceinline__ void fma2(float& d0, float& d1, float a0, float a1, float b) {
    asm("{\n\t.reg .b64 ra, rb, rd;\n\tmov.b64 ra, {%2, %3};\n\tmov.b64 rb, {%4, %4};\n\tmov.b64 rd, {%0, %1};\n\t"
        "fma.rn.f32x2 rd, ra, rb, rd;\n\tmov.b64 {%0, %1}, rd;\n\t}" : "+f"(d0), "+f"(d1) : "f"(a0), "f"(a1), "f"(b));
}
__device__ __forceinline__ void store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }

template <typename T>
__global__ void __launch_bounds__(MIXT) joint_qkv_store_kernel(const JointStoreArgs a) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float2 red[MIXT / 32];
    const int t = blockIdx.x, HD = a.H * a.D, GD = a.G * a.D, GV = a.G * a.Dv, per = a.H / a.G;
    const bool store = blockIdx.y == 0 && a.write_kv;                // one CTA of the token writes its keys and values
    const int h0 = blockIdx.y * a.heads_per_cta, h1 = min(a.H, h0 + a.heads_per_cta);
    float* ms = smem;                                                // [H][heads of this CTA, rounded up to HB]: mixing weights
    const int mh = (h1 - h0 + HB - 1) / HB * HB;
    float* qs = ms + a.H * mh;                                       // [H * D]
    float* ks = qs + HD;                                             // [G * D]
    for (int e = threadIdx.x; e < a.H * mh; e += MIXT) {             // (weights: not the predecessor's output)
        const int g = e / mh, h = h0 + (e - g * mh);
        ms[e] = h < h1 ? a.mix[(size_t)g * a.H + h] : 0.f;
    }
    TTIE_PDL_ENTRY();
    const T* row = reinterpret_cast<const T*>(a.proj) + (size_t)t * a.ld;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < HD; i += MIXT) { const float v = to_f32(row[i]); qs[i] = v; sq = fmaf(v, v, sq); }
    if (store) for (int i = threadIdx.x; i < GD; i += MIXT) { const float v = to_f32(row[HD + i]); ks[i] = v; sk = fmaf(v, v, sk); }
    if (a.norm_w) {
        const float2 ss = block_sum2(sq, sk, red);
        const float iq = 1.0f / sqrtf(ss.x / (float)HD + a.eps), ik = 1.0f / sqrtf(ss.y / (float)GD + a.eps);
        for (int i = threadIdx.x; i < HD; i += MIXT) qs[i] = qs[i] * iq * a.norm_w[i];
        if (store) for (int i = threadIdx.x; i < GD; i += MIXT) ks[i] = ks[i] * ik * a.norm_w[HD + i];
    }
    __syncthreads();
    if (a.rot > 0) {
        const float2* cs = a.cs + (size_t)t * (a.rot >> 1);
        rotate_rows(qs, a.H, a.D, a.rot, a.style, cs);
        if (store) rotate_rows(ks, a.G, a.D, a.rot, a.style, cs);
        __syncthreads();
    }
    if (store) {
        const int s = a.token_seq[t], pos = a.positions[t];
        int page = a.block_table[(size_t)s * a.table_width + pos / a.page_size];
        if (page < 0 || page >= a.num_pages) page = 0;               // validated on the host; never write outside
        const size_t dst = ((size_t)page * a.page_size + pos % a.page_size) * a.W;
        T* kp = reinterpret_cast<T*>(a.k_pages) + dst;
        T* vp = reinterpret_cast<T*>(a.v_pages) + dst;
        const T* vf = reinterpret_cast<const T*>(a.v_first);
        for (int i = threadIdx.x; i < a.W; i += MIXT) {
            kp[i] = from_f32<T>(i < GD ? ks[i] : 0.f);
            float v = 0.f;
            if (i < GV) {
                v = to_f32(row[HD + GD + i]);
                if (vf) v = (1.0f - a.v_mix) * v + a.v_mix * to_f32(vf[(size_t)t * a.ld_first + i]);
            }
            vp[i] = from_f32<T>(v);
        }
    }
    // the mixed query rows: thread = column of the joint row (two columns where heads have even sizes), HB output heads at a time
    T* q = reinterpret_cast<T*>(a.q_out) + (size_t)t * a.H * a.W;
    if (a.D % 2 == 0 && a.W % 2 == 0) {
        const int half = a.W >> 1, blocks = (h1 - h0 + HB - 1) / HB;
        for (int e = threadIdx.x; e < half * blocks; e += MIXT) {
            const int hb = e / half * HB, i = (e % half) * 2;
            const int c = i / a.D, d = i - c * a.D;                  // kv head of the columns
            float acc[2][HB];
#pragma unroll
            for (int k = 0; k < HB; ++k) acc[0][k] = acc[1][k] = 0.f;
            if (c < a.G) {
                const float* qc = qs + (size_t)c * per * a.D + d;
                const float* mc = ms + (size_t)c * per * mh + hb;
#pragma unroll 4
                for (int g = 0; g < per; ++g) {
                    const float2 qv = *reinterpret_cast<const float2*>(qc + g * a.D);
                    const float4 m0 = *reinterpret_cast<const float4*>(mc + g * mh), m1 = *reinterpret_cast<const float4*>(mc + g * mh + 4);
                    fma2(acc[0][0], acc[0][1], m0.x, m0.y, qv.x); fma2(acc[0][2], acc[0][3], m0.z, m0.w, qv.x);
                    fma2(acc[0][4], acc[0][5], m1.x, m1.y, qv.x); fma2(acc[0][6], acc[0][7], m1.z, m1.w, qv.x);
                    fma2(acc[1][0], acc[1][1], m0.x, m0.y, qv.y); fma2(acc[1][2], acc[1][3], m0.z, m0.w, qv.y);
                    fma2(acc[1][4], acc[1][5], m1.x, m1.y, qv.y); fma2(acc[1][6], acc[1][7], m1.z, m1.w, qv.y);
                }
            }
#pragma unroll
            for (int k = 0; k < HB; ++k)
                if (h0 + hb + k < h1) store2(q + (size_t)(h0 + hb + k) * a.W + i, acc[0][k], acc[1][k]);
        }
        return;
    }
    for (int i = threadIdx.x; i < a.W; i += MIXT) {
        const int c = i / a.D, d = i - c * a.D;                      // kv head of the column
        for (int hb = 0; hb < h1 - h0; hb += HB) {
            float acc[HB];
#pragma unroll
            for (int k = 0; k < HB; ++k) acc[k] = 0.f;
            if (c < a.G) {
                const float* qc = qs + (size_t)c * per * a.D + d;
                const float* mc = ms + (size_t)c * per * mh + hb;
                for (int g = 0; g < per; ++g) {
                    const float qv = qc[g * a.D];
                    const float4 m0 = *reinterpret_cast<const float4*>(mc + g * mh), m1 = *reinterpret_cast<const float4*>(mc + g * mh + 4);
                    acc[0] = fmaf(m0.x, qv, acc[0]); acc[1] = fmaf(m0.y, qv, acc[1]); acc[2] = fmaf(m0.z, qv, acc[2]); acc[3] = fmaf(m0.w, qv, acc[3]);
                    acc[4] = fmaf(m1.x, qv, acc[4]); acc[5] = fmaf(m1.y, qv, acc[5]); acc[6] = fmaf(m1.z, qv, acc[6]); acc[7] = fmaf(m1.w, qv, acc[7]);
                }
            }
#pragma unroll
            for (int k = 0; k < HB; ++k)
                if (h0 + hb + k < h1) q[(size_t)(h0 + hb + k) * a.W + i] = from_f32<T>(acc[k]);
        }
    }
}

template <typename T>
__global__ void joint_values_kernel(const T* __restrict__ attn, T* __restrict__ out, int T_, int H, int per, int Dv, int W) {
    TTIE_PDL_ENTRY();
    const int col = blockIdx.x * blockDim.x + threadIdx.x;           // grid: (columns of a token's output row, tokens)
    if (col >= H * Dv) return;
    const int h = col / Dv, j = col - h * Dv;
    for (size_t t = blockIdx.y; t < (size_t)T_; t += gridDim.y)
        out[t * H * Dv + col] = attn[(t * H + h) * W + (h / per) * Dv + j];
}

// eight bfloat16 per thread (value size and joint width multiples of 8, 16-byte aligned arrays)
__global__ void joint_values_vec8_kernel(const uint4* __restrict__ attn, uint4* __restrict__ out, int T_, int H, int per, int Dv8, int W8) {
    TTIE_PDL_ENTRY();
    const int col = blockIdx.x * blockDim.x + threadIdx.x;
    if (col >= H * Dv8) return;
    const int h = col / Dv8, j = col - h * Dv8;
    for (size_t t = blockIdx.y; t < (size_t)T_; t += gridDim.y)
        out[t * H * Dv8 + col] = attn[(t * H + h) * W8 + (h / per) * Dv8 + j];
}

size_t store_smem(int H, int G, int D, int heads_per_cta) {
    return ((size_t)H * ((heads_per_cta + HB - 1) / HB * HB) + (size_t)H * D + (size_t)G * D) * sizeof(float);
}
constexpr size_t STORE_SMEM = 220 * 1024;
}  // namespace

// 1 if joint_qkv_store takes these sizes (one token's query and key rows and HB columns of the mixing matrix in shared memory)
extern "C" int ttie_joint_store_supported(int H, int G, int D) { return store_smem(H, G, D, HB) <= STORE_SMEM ? 1 : 0; }

extern "C" int ttie_joint_qkv_store(const void* proj, long long ld, int T, int H, int G, int D, int Dv, int W, const float* mix,
                                    const float* norm_w, float eps, const void* cs, int rot, int style, const void* v_first,
                                    long long ld_first, float v_mix, const int* positions, const int* token_seq, const int* block_table,
                                    int table_width, int page_size, int num_pages, int write_kv, void* q_out, void* k_pages, void* v_pages,
                                    int dtype, void* stream) {
    if (T <= 0) return 0;
    if (G <= 0 || H % G) TTIE_FAIL("joint_qkv_store: %d heads are not a multiple of %d kv heads", H, G);
    if ((long long)G * D > W || (long long)G * Dv > W) TTIE_FAIL("joint_qkv_store: rows of %d values do not hold %d heads of %d / %d", W, G, D, Dv);
    if (rot < 0 || rot > D || rot % 2) TTIE_FAIL("joint_qkv_store: %d rotated values of a head of %d", rot, D);
    if (rot > 0 && !cs) TTIE_FAIL("joint_qkv_store: a rotation needs the step's cos/sin table");
    if (!mix) TTIE_FAIL("joint_qkv_store: no mixing matrix");
    JointStoreArgs a;
    a.proj = proj; a.ld = ld; a.H = H; a.G = G; a.D = D; a.Dv = Dv; a.W = W; a.mix = mix; a.norm_w = norm_w; a.eps = eps;
    a.cs = (const float2*)cs; a.rot = rot; a.style = style; a.v_first = v_first; a.ld_first = ld_first; a.v_mix = v_mix;
    a.positions = positions; a.token_seq = token_seq; a.block_table = block_table; a.table_width = table_width; a.page_size = page_size;
    a.num_pages = num_pages; a.write_kv = write_kv; a.q_out = q_out; a.k_pages = k_pages; a.v_pages = v_pages;
    // few tokens: the output heads of a token are shared out over CTAs (each reads the token's row again); many: one CTA per token
    int hpc = (H + HB - 1) / HB * HB;
    while (hpc > HB && ((long long)T * ceil_div(H, hpc) < num_sms() || store_smem(H, G, D, hpc) > STORE_SMEM)) hpc = (hpc / 2 + HB - 1) / HB * HB;
    a.heads_per_cta = hpc;
    const size_t smem = store_smem(H, G, D, hpc);
    if (smem > STORE_SMEM) TTIE_FAIL("joint_qkv_store: %d heads of %d values need %zu bytes of shared memory", H, D, smem);
    const dim3 grid(T, ceil_div(H, hpc));
    if (grid.y > 65535) TTIE_FAIL("joint_qkv_store: %d heads exceed the grid", H);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == kF32) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(joint_qkv_store_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        TTIE_LAUNCH(joint_qkv_store_kernel<float>, grid, MIXT, smem, s, a);
    } else if (dtype == kBF16) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(joint_qkv_store_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        TTIE_LAUNCH(joint_qkv_store_kernel<__nv_bfloat16>, grid, MIXT, smem, s, a);
    } else TTIE_FAIL("joint_qkv_store: unknown dtype %d", dtype);
    TTIE_CHECK_LAUNCH("joint_qkv_store");
    return 0;
}

extern "C" int ttie_joint_values(const void* attn, void* out, int T, int H, int G, int Dv, int W, int dtype, void* stream) {
    if (T <= 0) return 0;
    if (G <= 0 || H % G || (long long)G * Dv > W) TTIE_FAIL("joint_values: %d heads, %d kv heads of %d values in rows of %d", H, G, Dv, W);
    cudaStream_t s = (cudaStream_t)stream;
    const int per = H / G, rows = T < 65535 ? T : 65535;
    if (dtype == kBF16 && Dv % 8 == 0 && W % 8 == 0 && !(((uintptr_t)attn | (uintptr_t)out) & 15))
        TTIE_LAUNCH(joint_values_vec8_kernel, dim3(ceil_div(H * Dv / 8, 128), rows), 128, 0, s, (const uint4*)attn, (uint4*)out, T, H, per, Dv / 8, W / 8);
    else if (dtype == kBF16) TTIE_LAUNCH(joint_values_kernel<__nv_bfloat16>, dim3(ceil_div(H * Dv, 256), rows), 256, 0, s, (const __nv_bfloat16*)attn, (__nv_bfloat16*)out, T, H, per, Dv, W);
    else if (dtype == kF32) TTIE_LAUNCH(joint_values_kernel<float>, dim3(ceil_div(H * Dv, 256), rows), 256, 0, s, (const float*)attn, (float*)out, T, H, per, Dv, W);
    else TTIE_FAIL("joint_values: unknown dtype %d", dtype);
    TTIE_CHECK_LAUNCH("joint_values");
    return 0;
}
