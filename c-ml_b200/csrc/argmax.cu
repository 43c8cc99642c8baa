// Greedy pick over rows of logits, whole or split over ranks.
#include "lm_util.cuh"

namespace {

// ---- greedy pick: first index holding the strict maximum of each row
__device__ __forceinline__ void argmax_take(float& bv, int& bi, float v, int i) {
    if (v > bv || (v == bv && i < bi)) { bv = v; bi = i; }          // first index of the strict maximum; NaN never wins
}
__device__ __forceinline__ void argmax_warp(float& bv, int& bi) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
        const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
        argmax_take(bv, bi, ov, oi);
    }
}
// One cluster of ARGMAX_CTAS CTAs per row: every CTA scans a contiguous slice of the row with
// 16-byte loads, the slice winners meet in the shared memory of the cluster's first CTA
// (distributed shared memory), which picks the row's winner. No global scratch, fixed order.
constexpr int ARGMAX_CTAS = 8, ARGMAX_THREADS = 256;
__global__ void __cluster_dims__(ARGMAX_CTAS, 1, 1) __launch_bounds__(ARGMAX_THREADS)
argmax_kernel(const float* __restrict__ logits, int vocab, int* __restrict__ out, float2* __restrict__ out_pair, int index_offset) {
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    __shared__ float sv[ARGMAX_THREADS / 32];
    __shared__ int si[ARGMAX_THREADS / 32];
    __shared__ float cv[ARGMAX_CTAS];
    __shared__ int ci[ARGMAX_CTAS];
    const int part = blockIdx.x % ARGMAX_CTAS, r = blockIdx.x / ARGMAX_CTAS;
    const float* row = logits + (size_t)r * vocab;
    const int per = ((vocab + ARGMAX_CTAS - 1) / ARGMAX_CTAS + 3) & ~3;
    const int lo = min(vocab, part * per), hi = min(vocab, lo + per);
    float bv = -INFINITY;
    int bi = 0x7fffffff;
    if ((vocab & 3) == 0 && ((uintptr_t)row & 15) == 0) {
        for (int i = lo + threadIdx.x * 4; i < hi; i += ARGMAX_THREADS * 4) {
            const float4 v = *reinterpret_cast<const float4*>(row + i);
            argmax_take(bv, bi, v.x, i); argmax_take(bv, bi, v.y, i + 1);
            argmax_take(bv, bi, v.z, i + 2); argmax_take(bv, bi, v.w, i + 3);
        }
    } else {
        for (int i = lo + threadIdx.x; i < hi; i += ARGMAX_THREADS) argmax_take(bv, bi, row[i], i);
    }
    argmax_warp(bv, bi);
    if ((threadIdx.x & 31) == 0) { sv[threadIdx.x >> 5] = bv; si[threadIdx.x >> 5] = bi; }
    __syncthreads();
    if (threadIdx.x < 32) {
        bv = threadIdx.x < ARGMAX_THREADS / 32 ? sv[threadIdx.x] : -INFINITY;
        bi = threadIdx.x < ARGMAX_THREADS / 32 ? si[threadIdx.x] : 0x7fffffff;
        argmax_warp(bv, bi);
        if (threadIdx.x == 0) {                            // this slice's winner into slot `part` of CTA 0's arrays
            uint32_t dv, di;
            asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(dv) : "r"((uint32_t)__cvta_generic_to_shared(&cv[part])), "r"(0));
            asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(di) : "r"((uint32_t)__cvta_generic_to_shared(&ci[part])), "r"(0));
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(dv), "f"(bv) : "memory");
            asm volatile("st.shared::cluster.u32 [%0], %1;" ::"r"(di), "r"(bi) : "memory");
        }
    }
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    if (part == 0 && threadIdx.x < 32) {
        bv = threadIdx.x < ARGMAX_CTAS ? cv[threadIdx.x] : -INFINITY;
        bi = threadIdx.x < ARGMAX_CTAS ? ci[threadIdx.x] : 0x7fffffff;
        argmax_warp(bv, bi);
        if (threadIdx.x == 0) {
            if (out) out[r] = (bi == 0x7fffffff) ? 0 : bi;
            // (value, global index) of this slice of a vocabulary split over ranks; an empty result keeps -inf
            if (out_pair) out_pair[r] = make_float2(bv, __int_as_float(bi == 0x7fffffff ? 0x7fffffff : bi + index_offset));
        }
    }
}

// Winner per row among `parts` (value, index) candidates laid out [part][row]: greatest value, lowest
// index among equals (the candidates come from consecutive slices of one row, so this is the row's
// first strict maximum).
__global__ void argmax_merge_kernel(const float2* __restrict__ pairs, int parts, int rows, int* __restrict__ out) {
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int r = blockIdx.x * blockDim.x + threadIdx.x;
    if (r >= rows) return;
    float bv = -INFINITY;
    int bi = 0x7fffffff;
    for (int q = 0; q < parts; q++) {
        const float2 c = pairs[(size_t)q * rows + r];
        argmax_take(bv, bi, c.x, __float_as_int(c.y));
    }
    out[r] = (bi == 0x7fffffff) ? 0 : bi;
}

}  // namespace

extern "C" int cmlb200_argmax(const float* d_logits, int rows, int vocab, int* d_out, void* stream) {
    CMLB_REQUIRE(d_logits && d_out && rows > 0 && vocab > 0, "cmlb200_argmax: bad argument");
    CMLB_CUDA(launch_chain(argmax_kernel, dim3(rows * ARGMAX_CTAS), dim3(ARGMAX_THREADS), 0, 1, as_stream(stream), d_logits, vocab, d_out, (float2*)nullptr, 0));
    CMLB_LAUNCH_CHECK();
    return CMLB200_OK;
}

extern "C" int cmlb200_argmax_slice(const float* d_logits, int rows, int width, int index_offset, float* d_pairs, void* stream) {
    CMLB_REQUIRE(d_logits && d_pairs && rows > 0 && width > 0 && index_offset >= 0, "cmlb200_argmax_slice: bad argument");
    CMLB_CUDA(launch_chain(argmax_kernel, dim3(rows * ARGMAX_CTAS), dim3(ARGMAX_THREADS), 0, 1, as_stream(stream), d_logits, width, (int*)nullptr,
                         reinterpret_cast<float2*>(d_pairs), index_offset));
    CMLB_LAUNCH_CHECK();
    return CMLB200_OK;
}

extern "C" int cmlb200_argmax_merge(const float* d_pairs, int parts, int rows, int* d_out, void* stream) {
    CMLB_REQUIRE(d_pairs && d_out && parts > 0 && rows > 0, "cmlb200_argmax_merge: bad argument");
    CMLB_CUDA(launch_chain(argmax_merge_kernel, dim3((rows + 63) / 64), dim3(64), 0, 1, as_stream(stream), reinterpret_cast<const float2*>(d_pairs), parts, rows, d_out));
    CMLB_LAUNCH_CHECK();
    return CMLB200_OK;
}
