// Shared pieces of the layered-model kernels: programmatic dependent launches, reductions and the
// element conversions of the two number formats those models run in.
#pragma once
#include <cuda_fp16.h>
#include "common.cuh"

namespace {

// Every kernel of a step is launched so that it may become resident while its predecessor drains;
// each one waits here before it touches anything an earlier kernel of the stream wrote.
__device__ __forceinline__ void dep_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void dep_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

// cluster > 1: the grid's x dimension is cut into clusters of that many CTAs.
template <typename Kern, typename... Args>
cudaError_t launch_chain(Kern kern, dim3 grid, dim3 block, size_t smem, int cluster, cudaStream_t st, Args... args) {
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = (unsigned)cluster;
    attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = 1;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cfg.attrs = attr;
    cfg.numAttrs = cluster > 1 ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, kern, args...);
}

__device__ __forceinline__ float lane_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float lane_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}
// Sum over the block of up to 32 warps; `red` holds 32 floats and may be reused after the next barrier.
__device__ __forceinline__ float block_sum(float v, float* red) {
    v = lane_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
    for (int k = 0; k < (int)(blockDim.x >> 5); k++) t += red[k];
    return t;
}

// Two sums at once.
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* red) {
    a = lane_sum(a);
    b = lane_sum(b);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = make_float2(a, b);
    __syncthreads();
    float2 t = make_float2(0.f, 0.f);
    for (int k = 0; k < (int)(blockDim.x >> 5); k++) { t.x += red[k].x; t.y += red[k].y; }
    return t;
}
// This thread's share of the sum of squares of n floats; 16-byte loads where p allows them.
__device__ __forceinline__ float square_share(const float* p, int n) {
    float s = 0.f;
    if ((((uintptr_t)p | (unsigned)(n * 4)) & 15) == 0) {
#pragma unroll 4
        for (int i = threadIdx.x; i < (n >> 2); i += blockDim.x) {
            const float4 v = reinterpret_cast<const float4*>(p)[i];
            s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
        }
    } else {
#pragma unroll 4
        for (int i = threadIdx.x; i < n; i += blockDim.x) { const float v = p[i]; s = fmaf(v, v, s); }
    }
    return s;
}

__device__ __forceinline__ float widen(float v) { return v; }
__device__ __forceinline__ float widen(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float widen(__half v) { return __half2float(v); }
template <typename T> __device__ __forceinline__ T narrow(float v);
template <> __device__ __forceinline__ float narrow<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 narrow<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
// fp16 is only used for cached keys and values; anything beyond its range is held at its end
template <> __device__ __forceinline__ __half narrow<__half>(float v) { return __float2half_rn(fminf(fmaxf(v, -65504.f), 65504.f)); }

// tanh form of gelu: 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))
__device__ __forceinline__ float gelu_tanh(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sigmoidf(float z) { return 1.0f / (1.0f + expf(-z)); }
// 0.5 z (1 + erf(z / sqrt(2)))
__device__ __forceinline__ float gelu_erf(float z) { return 0.5f * z * (1.0f + erff(0.7071067811865476f * z)); }
__device__ __forceinline__ float unary_act(int act, float z) { return act == CMLB200_ACT_GELU_ERF ? gelu_erf(z) : (act == CMLB200_ACT_GELU_TANH ? gelu_tanh(z) : silu(z)); }
__device__ __forceinline__ float glu_act(int act, float g, float u, float limit = 0.f) {
    if (act == CMLB200_ACT_CLAMPED) {
        g = fminf(g, limit);
        return g * sigmoidf(1.702f * g) * (fminf(fmaxf(u, -limit), limit) + 1.0f);
    }
    return unary_act(act, g) * u;
}

// The same for results that are rounded to bf16: hardware exponential and reciprocal without branches, so that
// independent values overlap. The tanh form of gelu is z sigmoid(2 sqrt(2/pi) (z + 0.044715 z^3)).
__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
__device__ __forceinline__ float glu_act_fast(int act, float g, float u, float limit = 0.f) {
    const bool clamped = act == CMLB200_ACT_CLAMPED;
    g = clamped ? fminf(g, limit) : g;
    u = clamped ? fminf(fmaxf(u, -limit), limit) + 1.0f : u;
    const float gelu = 1.5957691216057308f * (g + 0.044715f * g * g * g);
    return g * sigmoid_fast(clamped ? 1.702f * g : (act == CMLB200_ACT_GELU_TANH ? gelu : g)) * u;
}

// erfc by the rational approximation 7.1.26 of Abramowitz and Stegun, Handbook of Mathematical Functions (error below 1.5e-7),
// so that nothing branches and nothing cancels on the negative side
__device__ __forceinline__ float gelu_erf_fast(float z) {
    const float x = fabsf(z) * 0.7071067811865476f, t = __fdividef(1.0f, fmaf(0.3275911f, x, 1.0f));
    float p = fmaf(1.061405429f, t, -1.453152027f);
    p = fmaf(p, t, 1.421413741f);
    p = fmaf(p, t, -0.284496736f);
    p = fmaf(p, t, 0.254829592f);
    const float tail = 0.5f * z * p * t * __expf(-x * x);
    return z > 0.f ? z - tail : tail;
}
// act: CMLB200_ACT_SILU, _GELU_TANH or _GELU_ERF
__device__ __forceinline__ float unary_act_fast(int act, float z) {
    if (act == CMLB200_ACT_GELU_ERF) return gelu_erf_fast(z);
    return z * sigmoid_fast(act == CMLB200_ACT_GELU_TANH ? 1.5957691216057308f * (z + 0.044715f * z * z * z) : z);
}

__device__ __forceinline__ float soft_cap(float v, float cap) { return cap * tanhf(v / cap); }

// Pieces of the mma.sync kernels.
constexpr float kLog2e = 1.4426950408889634f;
__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp16(uint32_t dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void mma_f16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ float ex2(float v) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
    return r;
}
// 16 bytes of a weight that is read once
__device__ __forceinline__ uint4 ld_stream(const __nv_bfloat16* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.L2::128B.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

}  // namespace
extern "C" int cmlb200_attn_check_(const cmlb200_attn* a, const char* who);
