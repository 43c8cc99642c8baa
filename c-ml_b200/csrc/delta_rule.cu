// Gated delta rule (see cmlb200_delta): a recurrence over tokens with one matrix of state per head, everything in fp32.
// With S read after the decay, s_k = S^T k and s_q = S^T q are sums over the same elements, and
//   u = beta (v - s_k),  o = s_q + (k . q) u,  S <- S + k u^T,
// so that a token needs one pass over S for both sums and one for the update.
//
//   delta_one_kernel      decoded tokens, one row per sequence: convolution, unit norms, decay, state, output norm and gate
//                         in one launch. A head's columns may be split over a cluster, which shares the output's square sum
//   delta_prepare_kernel  portions: convolutions, unit norms, decays, steps and k . q of all rows, a warp per head
//   delta_scan_kernel     portions: the recurrence. A CTA keeps 32 columns of a head's state in registers and walks the
//                         run's tokens, which arrive through a ring of shared memory; 8 lanes share a column
//   delta_output_kernel   portions: output norm and gate, a warp per (row, head)
//
// A sequence's latest projections lie in a ring of `taps` entries, position p in entry p mod taps: a token reads the
// entries before its own and writes its own, so the heads that share a key may do both in any order.
#include "lm_util.cuh"

namespace {

constexpr float kUnitEps = 1e-6f;

__device__ __forceinline__ int delta_channels(const cmlb200_delta& a) { return 2 * a.kv_heads * a.dim + a.heads * a.vdim; }
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float decay(const cmlb200_delta& a, int h, int i, float z) { return expf(-a.rate[h] * softplus(z + a.dt_bias[i])); }
__device__ __forceinline__ float delta_scale(const cmlb200_delta& a) { return a.out_scale == 0.f ? 1.f : a.out_scale; }

// Channel c at a row: the row's own projection and those of the tokens before it, from the rows in front (`back` of them belong to the
// same sequence's portion) or from the ring.
__device__ __forceinline__ float convolve(const cmlb200_delta& a, const float* __restrict__ proj, int ld, const float* __restrict__ ring, int channels, int c, int p,
                                          int back) {
    const float* x = proj + a.col + c;
    float y = a.conv[(size_t)(a.taps - 1) * channels + c] * x[0];
    for (int t = 1; t < a.taps && t <= p; t++) {
        const float v = t <= back ? x[-(ptrdiff_t)t * ld] : ring[(size_t)((p - t) % a.taps) * channels + c];
        y = fmaf(a.conv[(size_t)(a.taps - 1 - t) * channels + c], v, y);
    }
    return silu(y);
}

constexpr int ONE_THREADS = 256, ONE_WARPS = ONE_THREADS / 32;

// grid = (splits, heads, rows), clusters of `splits` CTAs along x. Thread (rg, c): four columns 4c of every `groups`-th row
// from rg on; RPT: room for those rows. lanes: threads across the columns of a CTA, a power of two.
template <typename TO, int RPT>
__global__ void __launch_bounds__(ONE_THREADS)
delta_one_kernel(const cmlb200_delta a, const float* __restrict__ proj, int ld, const float* __restrict__ dec, int ld_dec, const float* __restrict__ gate, int ld_gate,
                 const int* __restrict__ row_pos, const int* __restrict__ row_slot, int cols, int lanes, TO* __restrict__ out, int out_ld) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float2 red2[ONE_WARPS];
    __shared__ float red[ONE_WARPS], share;
    const int dimp = (a.dim + 3) & ~3;
    float *q_s = sm, *k_s = q_s + dimp, *g_s = k_s + dimp, *v_s = g_s + dimp, *part = v_s + cols;        // part: [8][lanes][8]
    const int splits = gridDim.x, rank = blockIdx.x, h = blockIdx.y, r = blockIdx.z;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int channels = delta_channels(a), group = a.heads / a.kv_heads, kh = h / group;
    const int c = tid & (lanes - 1), rg = tid / lanes, groups = ONE_THREADS / lanes, c0 = rank * cols + 4 * c;
    dep_wait();
    dep_trigger();
    const int p = row_pos[r], slot = row_slot[r];
    const float* row = proj + (size_t)r * ld;
    float* ring = a.ring + (size_t)slot * a.taps * channels;
    float4* state = reinterpret_cast<float4*>(a.state + ((size_t)slot * a.heads + h) * a.dim * a.vdim_ld + c0);
    const bool mine = 4 * c < cols && c0 < a.vdim_ld;
    float4 S[RPT];
#pragma unroll
    for (int i = 0; i < RPT; i++) {
        const int d = rg + i * groups;
        S[i] = mine && p > 0 && d < a.dim ? state[(size_t)d * (a.vdim_ld >> 2)] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float sq = 0.f, sk = 0.f;
    const bool keeps = rank == 0 && h == kh * group;
    for (int d = tid; d < a.dim; d += ONE_THREADS) {
        const int cq = kh * a.dim + d, ck = a.kv_heads * a.dim + cq;
        const float q = convolve(a, row, ld, ring, channels, cq, p, 0), k = convolve(a, row, ld, ring, channels, ck, p, 0);
        q_s[d] = q;
        k_s[d] = k;
        g_s[d] = decay(a, h, h * a.dim + d, dec[(size_t)r * ld_dec + h * a.dim + d]);
        sq = fmaf(q, q, sq);
        sk = fmaf(k, k, sk);
        if (keeps) {
            ring[(size_t)(p % a.taps) * channels + cq] = row[a.col + cq];
            ring[(size_t)(p % a.taps) * channels + ck] = row[a.col + ck];
        }
    }
    for (int j = tid; j < cols; j += ONE_THREADS) {
        const int d = rank * cols + j, cv = 2 * a.kv_heads * a.dim + h * a.vdim + d;
        v_s[j] = d < a.vdim ? convolve(a, row, ld, ring, channels, cv, p, 0) : 0.f;
        if (d < a.vdim) ring[(size_t)(p % a.taps) * channels + cv] = row[a.col + cv];
    }
    const float2 ss = block_sum2(sq, sk, red2);        // the barriers inside also publish q_s .. v_s
    const float iq = 1.0f / sqrtf(ss.x + kUnitEps) / sqrtf((float)a.dim), ik = 1.0f / sqrtf(ss.y + kUnitEps);
    const float beta = sigmoidf(row[a.col + channels + h]);
    float kq = 0.f;
    float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
#pragma unroll
    for (int i = 0; i < RPT; i++) {
        const int d = rg + i * groups;
        if (d >= a.dim) continue;
        const float k = k_s[d] * ik, q = q_s[d] * iq, g = g_s[d];
        kq = fmaf(k, q, kq);
        S[i].x *= g; S[i].y *= g; S[i].z *= g; S[i].w *= g;
        ak.x = fmaf(k, S[i].x, ak.x); ak.y = fmaf(k, S[i].y, ak.y); ak.z = fmaf(k, S[i].z, ak.z); ak.w = fmaf(k, S[i].w, ak.w);
        aq.x = fmaf(q, S[i].x, aq.x); aq.y = fmaf(q, S[i].y, aq.y); aq.z = fmaf(q, S[i].z, aq.z); aq.w = fmaf(q, S[i].w, aq.w);
    }
    // sums over the row groups: those of a warp by shuffles, the rest through shared memory
    for (int o = lanes; o < 32; o <<= 1) {
        ak.x += __shfl_xor_sync(0xffffffffu, ak.x, o); ak.y += __shfl_xor_sync(0xffffffffu, ak.y, o);
        ak.z += __shfl_xor_sync(0xffffffffu, ak.z, o); ak.w += __shfl_xor_sync(0xffffffffu, ak.w, o);
        aq.x += __shfl_xor_sync(0xffffffffu, aq.x, o); aq.y += __shfl_xor_sync(0xffffffffu, aq.y, o);
        aq.z += __shfl_xor_sync(0xffffffffu, aq.z, o); aq.w += __shfl_xor_sync(0xffffffffu, aq.w, o);
        kq += __shfl_xor_sync(0xffffffffu, kq, o);
    }
    float* kq_part = part + (size_t)8 * lanes * 8;     // [8]: a column's worth, the same for all columns
    const int pieces = lanes <= 32 ? ONE_WARPS : groups, piece = lanes <= 32 ? warp : rg;
    if (lanes > 32 || lane < lanes) {
        float4* dst = reinterpret_cast<float4*>(part + ((size_t)piece * lanes + c) * 8);
        dst[0] = ak;
        dst[1] = aq;
        if (c == 0) kq_part[piece] = kq;
    }
    __syncthreads();
    ak = make_float4(0.f, 0.f, 0.f, 0.f);
    aq = ak;
    kq = 0.f;
    for (int w = 0; w < pieces; w++) {
        const float4* src = reinterpret_cast<const float4*>(part + ((size_t)w * lanes + c) * 8);
        const float4 x = src[0], y = src[1];
        ak.x += x.x; ak.y += x.y; ak.z += x.z; ak.w += x.w;
        aq.x += y.x; aq.y += y.y; aq.z += y.z; aq.w += y.w;
        kq += kq_part[w];
    }
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f), o = u;
    if (mine) {
        const float4 v = make_float4(v_s[4 * c], v_s[4 * c + 1], v_s[4 * c + 2], v_s[4 * c + 3]);
        u = make_float4(beta * (v.x - ak.x), beta * (v.y - ak.y), beta * (v.z - ak.z), beta * (v.w - ak.w));
        o = make_float4(fmaf(kq, u.x, aq.x), fmaf(kq, u.y, aq.y), fmaf(kq, u.z, aq.z), fmaf(kq, u.w, aq.w));
    }
#pragma unroll
    for (int i = 0; i < RPT; i++) {
        const int d = rg + i * groups;
        if (!mine || d >= a.dim) continue;
        const float k = k_s[d] * ik;
        state[(size_t)d * (a.vdim_ld >> 2)] = make_float4(fmaf(k, u.x, S[i].x), fmaf(k, u.y, S[i].y), fmaf(k, u.z, S[i].z), fmaf(k, u.w, S[i].w));
    }
    float total = block_sum(rg == 0 ? fmaf(o.x, o.x, fmaf(o.y, o.y, fmaf(o.z, o.z, o.w * o.w))) : 0.f, red);
    if (splits > 1) {
        if (tid == 0) share = total;
        asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
        asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
        total = 0.f;
        for (int s = 0; s < splits; s++) {
            uint32_t at;
            float v;
            asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(at) : "r"(smem_addr(&share)), "r"(s));
            asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(at) : "memory");
            total += v;
        }
    }
    if (rg == 0 && mine) {
        const float inv = delta_scale(a) / sqrtf(total / (float)a.vdim + a.eps), os[4] = {o.x, o.y, o.z, o.w};
        TO* dst = out + (size_t)r * out_ld + h * a.vdim;
        const float* gr = gate + (size_t)r * ld_gate + h * a.vdim;
#pragma unroll
        for (int e = 0; e < 4; e++)
            if (c0 + e < a.vdim) dst[c0 + e] = narrow<TO>(os[e] * inv * a.norm[c0 + e] * sigmoidf(gr[c0 + e]));
    }
    if (splits > 1) {                                  // nobody leaves while others read its share
        asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
        asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    }
}

// A work row of a portion's token: [q (kv_heads dim) | k (kv_heads dim) | v, later o (heads vdim) | beta (heads) | k . q (kv_heads)].
__host__ __device__ inline int work_ld(const cmlb200_delta& a) { return (2 * a.kv_heads * a.dim + a.heads * a.vdim + a.heads + a.kv_heads + 3) & ~3; }

// grid = (rows, units / 8): a warp makes a key head's q and k, or a head's v, decays and step.
__global__ void __launch_bounds__(256)
delta_prepare_kernel(const cmlb200_delta a, const float* __restrict__ proj, int ld, float* __restrict__ dec, int ld_dec, const int* __restrict__ row_pos,
                     const int* __restrict__ row_slot, int first, float* __restrict__ work) {
    dep_wait();
    dep_trigger();
    const int r = first + blockIdx.x, unit = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= a.kv_heads + a.heads) return;
    const int channels = delta_channels(a), p = row_pos[r], slot = row_slot[r], kd = a.kv_heads * a.dim;
    int back = 0;                                      // rows right in front that belong to the same portion: a step has one per sequence
    while (back < a.taps - 1 && r - back - 1 >= first && row_slot[r - back - 1] == slot) back++;
    const float* row = proj + (size_t)r * ld;
    const float* ring = a.ring + (size_t)slot * a.taps * channels;
    float* w = work + (size_t)blockIdx.x * work_ld(a);
    if (unit < a.kv_heads) {
        float sq = 0.f, sk = 0.f, kq = 0.f, q[8], k[8];
#pragma unroll
        for (int i = 0; i < 8; i++) {                  // dim up to 256
            const int d = lane + 32 * i, c = unit * a.dim + d;
            q[i] = 0.f; k[i] = 0.f;
            if (d >= a.dim) continue;
            q[i] = convolve(a, row, ld, ring, channels, c, p, back);
            k[i] = convolve(a, row, ld, ring, channels, kd + c, p, back);
            sq = fmaf(q[i], q[i], sq);
            sk = fmaf(k[i], k[i], sk);
        }
        const float iq = 1.0f / sqrtf(lane_sum(sq) + kUnitEps) / sqrtf((float)a.dim), ik = 1.0f / sqrtf(lane_sum(sk) + kUnitEps);
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int d = lane + 32 * i;
            if (d >= a.dim) continue;
            q[i] *= iq;
            k[i] *= ik;
            kq = fmaf(k[i], q[i], kq);
            w[unit * a.dim + d] = q[i];
            w[kd + unit * a.dim + d] = k[i];
        }
        kq = lane_sum(kq);
        if (lane == 0) w[channels + a.heads + unit] = kq;
        return;
    }
    const int h = unit - a.kv_heads;
    for (int d = lane; d < a.vdim; d += 32) {
        const int c = 2 * kd + h * a.vdim + d;
        w[c] = convolve(a, row, ld, ring, channels, c, p, back);
    }
    float* g = dec + (size_t)r * ld_dec + h * a.dim;
    for (int d = lane; d < a.dim; d += 32) g[d] = decay(a, h, h * a.dim + d, g[d]);
    if (lane == 0) w[channels + h] = sigmoidf(row[a.col + channels + h]);
}

__device__ __forceinline__ uint64_t pack2(float x, float y) {
    uint64_t v;
    asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(x), "f"(y));
    return v;
}
__device__ __forceinline__ float sum2(uint64_t v) {
    float x, y;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(v));
    return x + y;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t v;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(v) : "l"(a), "l"(b), "l"(c));
    return v;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t v;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(v) : "l"(a), "l"(b));
    return v;
}
template <int N> __device__ __forceinline__ void copy_async(float* dst, const float* src) {
    if (N == 4) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
}

constexpr int SCAN_THREADS = 128, SCAN_COLS = 32;

// grid = (column slices, heads, runs). Lane (rg, cl) of a warp: rows 32 i + 4 rg .. + 3 of two columns; pairs of neighbouring
// rows share a register pair. RPL: rows per lane, a multiple of 4. N: floats per copy.
template <int RPL, int N>
__global__ void __launch_bounds__(SCAN_THREADS)
delta_scan_kernel(const cmlb200_delta a, const float* __restrict__ proj, int ld, const float* __restrict__ dec, int ld_dec, const int* __restrict__ row_pos,
                  const int4* __restrict__ runs, int first, float* __restrict__ work) {
    constexpr int DIM = RPL * 8, SCAN_TOKENS = RPL > 16 ? 4 : 8;       // tokens per stage
    __shared__ __align__(16) float ks[2][SCAN_TOKENS][DIM], qs[2][SCAN_TOKENS][DIM], gs[2][SCAN_TOKENS][DIM], vs[2][SCAN_TOKENS][SCAN_COLS];
    __shared__ float bs[2][SCAN_TOKENS], kqs[2][SCAN_TOKENS];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rg = lane >> 2, cl = lane & 3;
    const int h = blockIdx.y, group = a.heads / a.kv_heads, kh = h / group, channels = delta_channels(a), wld = work_ld(a);
    const int col0 = blockIdx.x * SCAN_COLS, mycol = col0 + warp * 8 + cl * 2;
    for (int i = tid; i < 2 * SCAN_TOKENS * DIM; i += SCAN_THREADS) { (&ks[0][0][0])[i] = 0.f; (&qs[0][0][0])[i] = 0.f; (&gs[0][0][0])[i] = 0.f; }
    for (int i = tid; i < 2 * SCAN_TOKENS * SCAN_COLS; i += SCAN_THREADS) (&vs[0][0][0])[i] = 0.f;
    dep_wait();
    dep_trigger();
    const int4 run = runs[blockIdx.z];
    const int r0 = run.x, n = run.y, slot = run.z, p0 = row_pos[r0];
    float* o = work + (size_t)(r0 - first) * wld + 2 * a.kv_heads * a.dim + h * a.vdim;
    __syncthreads();                                   // the zeros behind dim and vdim are in place
    auto fetch = [&](int b) {
        const int t0 = b * SCAN_TOKENS, st = b & 1, kd = a.dim / N, kv = min(SCAN_COLS, a.vdim - col0) / N;
        for (int i = tid; i < SCAN_TOKENS * kd; i += SCAN_THREADS) {
            const int t = i / kd, d = (i - t * kd) * N;
            if (t0 + t >= n) break;
            const float* w = work + (size_t)(r0 - first + t0 + t) * wld + kh * a.dim + d;
            copy_async<N>(&qs[st][t][d], w);
            copy_async<N>(&ks[st][t][d], w + a.kv_heads * a.dim);
            copy_async<N>(&gs[st][t][d], dec + (size_t)(r0 + t0 + t) * ld_dec + h * a.dim + d);
        }
        for (int i = tid; i < SCAN_TOKENS * kv; i += SCAN_THREADS) {
            const int t = i / kv, d = (i - t * kv) * N;
            if (t0 + t >= n) break;
            copy_async<N>(&vs[st][t][d], o + (size_t)(t0 + t) * wld + col0 + d);
        }
        if (tid < 2 * SCAN_TOKENS) {
            const int t = tid >> 1;
            if (t0 + t < n) {
                const float* w = work + (size_t)(r0 - first + t0 + t) * wld + channels;
                if (tid & 1) copy_async<1>(&kqs[st][t], w + a.heads + kh);
                else copy_async<1>(&bs[st][t], w + h);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0);
    uint64_t S[2][RPL / 2];
    float* state = a.state + ((size_t)slot * a.heads + h) * a.dim * a.vdim_ld;
#pragma unroll
    for (int i = 0; i < RPL / 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
            const int d = i * 32 + rg * 4 + j;
            const bool c_ok = mycol < a.vdim_ld && p0 > 0;              // vdim_ld is a multiple of 4 and mycol is even
            const float2 z = make_float2(0.f, 0.f);
            const float2 x = c_ok && d < a.dim ? *reinterpret_cast<const float2*>(state + (size_t)d * a.vdim_ld + mycol) : z;
            const float2 y = c_ok && d + 1 < a.dim ? *reinterpret_cast<const float2*>(state + (size_t)(d + 1) * a.vdim_ld + mycol) : z;
            S[0][i * 2 + j / 2] = pack2(x.x, y.x);
            S[1][i * 2 + j / 2] = pack2(x.y, y.y);
        }
    if (blockIdx.x == 0) {                             // the latest projections; nobody reads the ring in this launch
        const int keep = min(n, a.taps - 1), kd = a.kv_heads * a.dim;
        for (int t = n - keep; t < n; t++) {
            float* ring = a.ring + ((size_t)slot * a.taps + (p0 + t) % a.taps) * channels;
            const float* row = proj + (size_t)(r0 + t) * ld + a.col;
            if (h == kh * group)
                for (int d = tid; d < a.dim; d += SCAN_THREADS) {
                    ring[kh * a.dim + d] = row[kh * a.dim + d];
                    ring[kd + kh * a.dim + d] = row[kd + kh * a.dim + d];
                }
            for (int d = tid; d < a.vdim; d += SCAN_THREADS) ring[2 * kd + h * a.vdim + d] = row[2 * kd + h * a.vdim + d];
        }
    }
    const int blocks = (n + SCAN_TOKENS - 1) / SCAN_TOKENS;
    for (int b = 0; b < blocks; b++) {
        if (b + 1 < blocks) {
            fetch(b + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const int st = b & 1, tokens = min(SCAN_TOKENS, n - b * SCAN_TOKENS);
        for (int t = 0; t < tokens; t++) {
            const ulonglong2 *k4 = reinterpret_cast<const ulonglong2*>(ks[st][t]), *q4 = reinterpret_cast<const ulonglong2*>(qs[st][t]), *g4 = reinterpret_cast<const ulonglong2*>(gs[st][t]);
            uint64_t k[RPL / 2], ak[2][2] = {}, aq[2][2] = {};
#pragma unroll
            for (int i = 0; i < RPL / 4; i++) {
                const ulonglong2 g = g4[i * 8 + rg], kk = k4[i * 8 + rg], qq = q4[i * 8 + rg];
                k[2 * i] = kk.x;
                k[2 * i + 1] = kk.y;
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    S[c][2 * i] = mul2(S[c][2 * i], g.x);
                    S[c][2 * i + 1] = mul2(S[c][2 * i + 1], g.y);
                    ak[c][0] = fma2(S[c][2 * i], kk.x, ak[c][0]);
                    ak[c][1] = fma2(S[c][2 * i + 1], kk.y, ak[c][1]);
                    aq[c][0] = fma2(S[c][2 * i], qq.x, aq[c][0]);
                    aq[c][1] = fma2(S[c][2 * i + 1], qq.y, aq[c][1]);
                }
            }
            float sk[2], sq[2];
#pragma unroll
            for (int c = 0; c < 2; c++) { sk[c] = sum2(ak[c][0]) + sum2(ak[c][1]); sq[c] = sum2(aq[c][0]) + sum2(aq[c][1]); }
#pragma unroll
            for (int x = 4; x < 32; x <<= 1) {
#pragma unroll
                for (int c = 0; c < 2; c++) { sk[c] += __shfl_xor_sync(0xffffffffu, sk[c], x); sq[c] += __shfl_xor_sync(0xffffffffu, sq[c], x); }
            }
            const float2 v = *reinterpret_cast<const float2*>(&vs[st][t][warp * 8 + cl * 2]);
            const float beta = bs[st][t], kq = kqs[st][t], u0 = beta * (v.x - sk[0]), u1 = beta * (v.y - sk[1]);
            const uint64_t uu0 = pack2(u0, u0), uu1 = pack2(u1, u1);
#pragma unroll
            for (int i = 0; i < RPL / 2; i++) { S[0][i] = fma2(k[i], uu0, S[0][i]); S[1][i] = fma2(k[i], uu1, S[1][i]); }
            if (rg == 0) {
                float* dst = o + (size_t)(b * SCAN_TOKENS + t) * wld + mycol;
                if (mycol < a.vdim) dst[0] = fmaf(kq, u0, sq[0]);
                if (mycol + 1 < a.vdim) dst[1] = fmaf(kq, u1, sq[1]);
            }
        }
        __syncthreads();                               // this stage may be refilled
    }
#pragma unroll
    for (int i = 0; i < RPL / 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
            const int d = i * 32 + rg * 4 + j;
            float x0, x1, y0, y1;
            asm("mov.b64 {%0, %1}, %2;" : "=f"(x0), "=f"(y0) : "l"(S[0][i * 2 + j / 2]));
            asm("mov.b64 {%0, %1}, %2;" : "=f"(x1), "=f"(y1) : "l"(S[1][i * 2 + j / 2]));
            if (mycol < a.vdim_ld && d < a.dim) *reinterpret_cast<float2*>(state + (size_t)d * a.vdim_ld + mycol) = make_float2(x0, x1);
            if (mycol < a.vdim_ld && d + 1 < a.dim) *reinterpret_cast<float2*>(state + (size_t)(d + 1) * a.vdim_ld + mycol) = make_float2(y0, y1);
        }
}

template <typename TO>
__global__ void __launch_bounds__(256)
delta_output_kernel(const cmlb200_delta a, const float* __restrict__ work, const float* __restrict__ gate, int ld_gate, int first, TO* __restrict__ out, int out_ld) {
    dep_wait();
    dep_trigger();
    const int h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, r = first + blockIdx.x;
    if (h >= a.heads) return;
    const float* o = work + (size_t)blockIdx.x * work_ld(a) + 2 * a.kv_heads * a.dim + h * a.vdim;
    const float* g = gate + (size_t)r * ld_gate + h * a.vdim;
    float v[8], ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) {                      // vdim up to 256
        const int d = lane + 32 * i;
        v[i] = d < a.vdim ? o[d] : 0.f;
        ss = fmaf(v[i], v[i], ss);
    }
    const float inv = delta_scale(a) / sqrtf(lane_sum(ss) / (float)a.vdim + a.eps);
#pragma unroll
    for (int i = 0; i < 8; i++) {
        const int d = lane + 32 * i;
        if (d < a.vdim) out[(size_t)r * out_ld + h * a.vdim + d] = narrow<TO>(v[i] * inv * a.norm[d] * sigmoidf(g[d]));
    }
}

int delta_check(const cmlb200_delta* a, const float* proj, int ld, const float* dec, int ld_dec, const float* gate, int ld_gate, const int* pos, const int* slot,
                int rows, void* out, int out_dtype, int out_ld, const char* who) {
    CMLB_REQUIRE(a && proj && dec && gate && pos && slot && out && rows > 0 && rows <= 65535, "%s: bad argument", who);
    CMLB_REQUIRE(a->heads > 0 && a->heads <= 65535 && a->kv_heads > 0 && a->heads % a->kv_heads == 0 && a->dim > 0 && a->dim <= 256 && a->vdim > 0 && a->vdim <= 256 &&
                 a->taps > 0, "%s: heads %d, kv_heads %d, sizes %d / %d (up to 256), taps %d", who, a->heads, a->kv_heads, a->dim, a->vdim, a->taps);
    CMLB_REQUIRE(a->vdim_ld >= a->vdim && a->vdim_ld % 4 == 0 && a->state && a->ring && a->conv && a->rate && a->dt_bias && a->norm && ((uintptr_t)a->state & 15) == 0,
                 "%s: no state or weights", who);
    CMLB_REQUIRE(a->col >= 0 && ld >= a->col + 2 * a->kv_heads * a->dim + a->heads * (a->vdim + 1) && ld_dec >= a->heads * a->dim && ld_gate >= a->heads * a->vdim &&
                 out_ld >= a->heads * a->vdim, "%s: strides %d / %d / %d / %d", who, ld, ld_dec, ld_gate, out_ld);
    CMLB_REQUIRE(out_dtype == CMLB200_DT_F32 || out_dtype == CMLB200_DT_BF16, "%s: dtype %d", who, out_dtype);
    return CMLB200_OK;
}

}  // namespace

extern "C" int cmlb200_delta_one(const cmlb200_delta* a, const float* d_proj, int ld, const float* d_decay, int ld_decay, const float* d_gate, int ld_gate,
                                 const int* d_row_pos, const int* d_row_slot, int rows, void* d_out, int out_dtype, int out_ld, void* stream) {
    const int rc = delta_check(a, d_proj, ld, d_decay, ld_decay, d_gate, ld_gate, d_row_pos, d_row_slot, rows, d_out, out_dtype, out_ld, "cmlb200_delta_one");
    if (rc) return rc;
    // split the columns while that gives the SMs something to do, and until a thread's rows fit its registers
    auto shape = [&](int splits, int& cols, int& lanes) {
        cols = ((a->vdim + splits - 1) / splits + 3) & ~3;
        lanes = 4;
        while (lanes * 4 < cols) lanes *= 2;
        return (a->dim + ONE_THREADS / lanes - 1) / (ONE_THREADS / lanes);
    };
    int splits = 1, cols, lanes, rpt = shape(1, cols, lanes);
    while (splits < 8 && cols > 16 && (rpt > 16 || (long long)rows * a->heads * splits < 2 * cmlb_num_sms())) rpt = shape(splits *= 2, cols, lanes);
    CMLB_REQUIRE(rpt <= 32, "cmlb200_delta_one: states of %d x %d", a->dim, a->vdim);
    const size_t smem = sizeof(float) * ((size_t)3 * ((a->dim + 3) & ~3) + cols + (size_t)8 * lanes * 8 + 8);
    const dim3 grid(splits, a->heads, rows);
#define DO_LAUNCH(TO, RPT) CMLB_CUDA(launch_chain(delta_one_kernel<TO, RPT>, grid, dim3(ONE_THREADS), smem, splits, as_stream(stream), *a, d_proj, ld, d_decay, ld_decay, \
                                                  d_gate, ld_gate, d_row_pos, d_row_slot, cols, lanes, (TO*)d_out, out_ld))
#define DO_ROWS(TO) do { if (rpt <= 4) DO_LAUNCH(TO, 4); else if (rpt <= 8) DO_LAUNCH(TO, 8); else if (rpt <= 16) DO_LAUNCH(TO, 16); else DO_LAUNCH(TO, 32); } while (0)
    if (out_dtype == CMLB200_DT_BF16) DO_ROWS(__nv_bfloat16);
    else DO_ROWS(float);
#undef DO_ROWS
#undef DO_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_delta_work_floats(const cmlb200_delta* a) { return a ? work_ld(*a) : 0; }

extern "C" int cmlb200_delta_rows(const cmlb200_delta* a, const float* d_proj, int ld, float* d_decay, int ld_decay, const float* d_gate, int ld_gate,
                                  const int* d_row_pos, const int* d_row_slot, int first, int rows, const int* d_runs, int runs, float* d_work, void* d_out,
                                  int out_dtype, int out_ld, void* stream) {
    const int rc = delta_check(a, d_proj, ld, d_decay, ld_decay, d_gate, ld_gate, d_row_pos, d_row_slot, 1, d_out, out_dtype, out_ld, "cmlb200_delta_rows");
    if (rc) return rc;
    CMLB_REQUIRE(d_runs && runs > 0 && runs <= 65535 && rows > 0 && first >= 0 && d_work && (((uintptr_t)d_runs | (uintptr_t)d_work) & 15) == 0, "cmlb200_delta_rows: bad argument");
    cudaStream_t st = as_stream(stream);
    CMLB_CUDA(launch_chain(delta_prepare_kernel, dim3(rows, (a->kv_heads + a->heads + 7) / 8), dim3(256), 0, 1, st, *a, d_proj, ld, d_decay, ld_decay, d_row_pos, d_row_slot,
                           first, d_work));
    const bool vec = a->dim % 4 == 0 && a->vdim % 4 == 0 && ld_decay % 4 == 0 && ((uintptr_t)d_decay & 15) == 0;
    const dim3 grid((a->vdim + SCAN_COLS - 1) / SCAN_COLS, a->heads, runs);
#define DS_LAUNCH(RPL, N) CMLB_CUDA(launch_chain(delta_scan_kernel<RPL, N>, grid, dim3(SCAN_THREADS), 0, 1, st, *a, d_proj, ld, (const float*)d_decay, ld_decay, d_row_pos, \
                                                 (const int4*)d_runs, first, d_work))
#define DS_COPY(RPL) do { if (vec) DS_LAUNCH(RPL, 4); else DS_LAUNCH(RPL, 1); } while (0)
    if (a->dim <= 32) DS_COPY(4);
    else if (a->dim <= 64) DS_COPY(8);
    else if (a->dim <= 128) DS_COPY(16);
    else DS_COPY(32);
#undef DS_COPY
#undef DS_LAUNCH
    const dim3 grid_out(rows, (a->heads + 7) / 8);
    if (out_dtype == CMLB200_DT_BF16)
        CMLB_CUDA(launch_chain(delta_output_kernel<__nv_bfloat16>, grid_out, dim3(256), 0, 1, st, *a, (const float*)d_work, d_gate, ld_gate, first, (__nv_bfloat16*)d_out, out_ld));
    else
        CMLB_CUDA(launch_chain(delta_output_kernel<float>, grid_out, dim3(256), 0, 1, st, *a, (const float*)d_work, d_gate, ld_gate, first, (float*)d_out, out_ld));
    return CMLB200_OK;
}
