// Attention of a step's rows over paged caches, for layers described by a cmlb200_attn: grouped heads
// with separate query/key and value sizes, a sliding window or chunks (with or without the sequence's first
// tokens kept in sight), a per-head linear distance bias, a sink (one, or a learned exponential per head, added
// to the softmax denominator), norms over all heads or per head, rotated queries and keys, values that are the keys before their
// norm, scores that another kernel has made (talk_scores.cu), a per-head output gate. Rows of different sequences share a launch; every row finds its keys through its
// sequence's block table.
//
//   attention_tiles_kernel   prompt portions: 64 consecutive query rows of one sequence and one head per
//                            CTA, key tiles of 64 (only those some row's window reaches) double-buffered
//                            with cp.async, S = Q K^T and O += P V on mma.sync m16n8k16 (fp16 operands,
//                            fp32 scores, weights and sums)
//   attention_one_kernel     decoded tokens, one row per sequence: query/key norm, temperature, cache
//                            append, attention and gate in one launch. A cluster of up to 8 CTAs splits
//                            the keys of one (row, key/value head) and merges through distributed
//                            shared memory
//   attention_rows_f32_kernel  fp32 caches, one CTA per (row, head), everything in fp32
//
// Scores are kept in units of log2 in the first two kernels (the scale carries log2 e). A sink starts
// the running maximum at its score, so its weight joins the denominator exactly once.
#include "lm_util.cuh"

namespace {

__device__ __forceinline__ uint32_t pack_h2(float lo, float hi) {
    const __half2 v = __floats2half2_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}
constexpr int QT = 64, KT = 64, TILE_THREADS = 128;

// The first key that the row at position p sees, the kept ones (0 .. keep - 1) aside.
__device__ __forceinline__ int first_key(const cmlb200_attn& a, int p) {
    if (a.chunk > 0) return p / a.chunk * a.chunk;
    return (a.window > 0 && a.window <= p) ? p - a.window + 1 : 0;
}
__device__ __forceinline__ float sink_score(const cmlb200_attn& a, int h) { return a.sinks ? a.sinks[h] : 0.f; }
__device__ __forceinline__ float out_scale(const cmlb200_attn& a) { return a.out_scale == 0.f ? 1.f : a.out_scale; }

// grid = (tiles, heads). tiles[i] = {first row, rows (1..64), sequence slot, position of the first row}.
// DV: room for value columns. DK: 0, or the padded key size, and then DV is the padded value size. SCORED: scores come from
// a.scores, so there are neither queries nor keys.
template <int DV, int DK, bool SCORED>
__global__ void __launch_bounds__(TILE_THREADS)
attention_tiles_kernel(const cmlb200_attn a, const float* __restrict__ qkv, int ld, const int4* __restrict__ tiles, __nv_bfloat16* __restrict__ out,
                       int out_ld) {
    extern __shared__ __align__(16) __half sm[];
    const int dk = DK ? DK : a.dim_ld, dv = DK ? DV : a.vdim_ld, LK = dk + 8, LV = dv + 8;
    __half* Qs = sm;
    __half* Ks = Qs + (SCORED ? 0 : QT * LK);          // two stages each
    __half* Vs = Ks + (SCORED ? 0 : 2 * KT * LK);
    dep_wait();
    dep_trigger();
    const int4 tl = tiles[blockIdx.x];
    const int n = tl.y, p0 = tl.w, h = blockIdx.y, kh = h / (a.heads / a.kv_heads);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
    const int shift = __ffs(a.block_size) - 1;
    const int* table = a.block_table + (size_t)tl.z * a.table_ld;
    const int p_last = p0 + n - 1;
    // key tiles: those of the kept tokens, then from k_lo on (one run from 0 where they meet)
    int k_lo = first_key(a, p0) & ~15, kept_tiles = (min(a.keep, k_lo) + KT - 1) / KT;
    if (kept_tiles * KT >= k_lo) { k_lo = 0; kept_tiles = 0; }
    const int ntiles = kept_tiles + (p_last - k_lo) / KT + 1;
    auto tile_start = [&](int it) { return it < kept_tiles ? it * KT : k_lo + (it - kept_tiles) * KT; };
    const __half* kp = static_cast<const __half*>(a.k_pool) + (size_t)kh * dk;
    const __half* vp = static_cast<const __half*>(a.v_pool) + (size_t)kh * dv;
    const int kstride = a.kv_heads * dk, vstride = a.kv_heads * dv;

    auto load = [&](int it) {
        const int kt = tile_start(it), st = it & 1;
        const int kc = dk >> 3, vc = dv >> 3;
        for (int row = threadIdx.x >> 3; row < KT; row += TILE_THREADS / 8) {
            const int key = min(kt + row, p_last);     // rows past the end repeat the last key (masked below)
            const size_t slot = ((size_t)table[key >> shift] << shift) + (key & (a.block_size - 1));
            if (!SCORED)
                for (int c = threadIdx.x & 7; c < kc; c += 8) cp16(smem_addr(Ks + (st * KT + row) * LK + c * 8), kp + slot * kstride + c * 8);
            for (int c = threadIdx.x & 7; c < vc; c += 8) cp16(smem_addr(Vs + (st * KT + row) * LV + c * 8), vp + slot * vstride + c * 8);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load(0);
    if (!SCORED) {
        const float qs = a.scale * kLog2e;
        for (int r = warp; r < QT; r += TILE_THREADS / 32) {
            const float* src = qkv + (size_t)(tl.x + min(r, n - 1)) * ld + h * a.dim;
#pragma unroll 4
            for (int d = lane; d < dk; d += 32) Qs[r * LK + d] = d < a.dim ? narrow<__half>(src[d] * qs) : __float2half_rn(0.f);
        }
    }
    const float slope = a.slopes ? a.slopes[h] * kLog2e : 0.f;
    const int r0 = warp * 16 + g, r1 = r0 + 8;
    const int q0 = r0 < n ? p0 + r0 : -1, q1 = r1 < n ? p0 + r1 : -1;         // -1: sees nothing
    const int w_first = p0 + warp * 16, w_last = min(p0 + warp * 16 + 15, p_last);
    const int lo0 = first_key(a, max(q0, 0)), lo1 = first_key(a, max(q1, 0)), w_lo = first_key(a, w_first), w_lo_last = first_key(a, max(w_last, 0));
    const float sink = a.sink ? sink_score(a, h) * kLog2e : -INFINITY;
    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; i++) { o[i][0] = 0.f; o[i][1] = 0.f; o[i][2] = 0.f; o[i][3] = 0.f; }
    float m0 = sink, m1 = m0, l0 = 0.f, l1 = 0.f;
    // score of key kt + c from position q: dot - slope (q - kt - c). The part that depends on the column alone
    // is what the accumulators start from; the rest is one constant per row and tile.
    float bias[KT / 8][2];
#pragma unroll
    for (int i = 0; i < KT / 8; i++) { bias[i][0] = slope * (float)(i * 8 + 2 * t); bias[i][1] = slope * (float)(i * 8 + 2 * t + 1); }
    const uint32_t q_base = smem_addr(Qs + (warp * 16 + (lane & 15)) * LK + (lane >> 4) * 8);
    const float* scores = SCORED ? a.scores + (((size_t)blockIdx.x * a.heads + h) * QT + r0) * a.scores_ld : nullptr;

    for (int it = 0; it < ntiles; it++) {
        if (it + 1 < ntiles) {
            load(it + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const int kt = tile_start(it), st = it & 1;
        // nothing of this tile is in reach of this warp's rows: before all they see, or past the last row
        const bool active = w_first <= w_last && kt <= w_last && (kt + KT - 1 >= w_lo || kt < a.keep);
        if (active) {
            float s[KT / 8][4];
#pragma unroll
            for (int i = 0; i < KT / 8; i++) { s[i][0] = bias[i][0]; s[i][1] = bias[i][1]; s[i][2] = bias[i][0]; s[i][3] = bias[i][1]; }
            if constexpr (SCORED) {
                const float* src = scores + kt - k_lo + 2 * t;
#pragma unroll
                for (int i = 0; i < KT / 8; i++) {
                    const float2 x = *reinterpret_cast<const float2*>(src + i * 8), y = *reinterpret_cast<const float2*>(src + (size_t)8 * a.scores_ld + i * 8);
                    s[i][0] += x.x; s[i][1] += x.y; s[i][2] += y.x; s[i][3] += y.y;
                }
            } else {
                const uint32_t k_base = smem_addr(Ks + (st * KT + (lane & 7) + ((lane >> 4) & 1) * 8) * LK + ((lane >> 3) & 1) * 8);
#pragma unroll (DK ? DK / 16 : 1)
                for (int kk = 0; kk < dk; kk += 16) {
                    uint32_t qa[4];
                    ldsm4(q_base + kk * 2, qa);
#pragma unroll
                    for (int j = 0; j < KT / 16; j++) {
                        uint32_t b[4];
                        ldsm4(k_base + (j * 16 * LK + kk) * 2, b);
                        mma_f16(s[2 * j], qa, b[0], b[1]);
                        mma_f16(s[2 * j + 1], qa, b[2], b[3]);
                    }
                }
            }
            // unless every row of the warp sees every key of the tile
            if (!(kt + KT - 1 <= w_first && kt >= w_lo_last) || w_last - w_first < 15) {
#pragma unroll
                for (int i = 0; i < KT / 8; i++) {
#pragma unroll
                    for (int e = 0; e < 2; e++) {
                        const int key = kt + i * 8 + 2 * t + e;
                        const bool kept_key = key < a.keep;
                        if (key > q0 || (key < lo0 && !kept_key)) s[i][e] = -INFINITY;
                        if (key > q1 || (key < lo1 && !kept_key)) s[i][2 + e] = -INFINITY;
                    }
                }
            }
            float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
            for (int i = 0; i < KT / 8; i++) {
                mx0 = fmaxf(mx0, fmaxf(s[i][0], s[i][1]));
                mx1 = fmaxf(mx1, fmaxf(s[i][2], s[i][3]));
            }
            mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1)); mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1)); mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
            const float f0 = slope * (float)(kt - q0), f1 = slope * (float)(kt - q1);
            mx0 = fmaxf(m0, mx0 + f0);
            mx1 = fmaxf(m1, mx1 + f1);
            const float u0 = mx0 == -INFINITY ? 0.f : mx0, u1 = mx1 == -INFINITY ? 0.f : mx1;      // a row that has seen nothing yet
            const float c0 = ex2(m0 - u0), c1 = ex2(m1 - u1), g0 = u0 - f0, g1 = u1 - f1;
            m0 = mx0; m1 = mx1;
            l0 *= c0; l1 *= c1;
            if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
                for (int i = 0; i < DV / 8; i++) { o[i][0] *= c0; o[i][1] *= c0; o[i][2] *= c1; o[i][3] *= c1; }
            }
            uint32_t pa[KT / 16][4];
#pragma unroll
            for (int i = 0; i < KT / 8; i++) {
                const float e0 = ex2(s[i][0] - g0), e1 = ex2(s[i][1] - g0), e2 = ex2(s[i][2] - g1), e3 = ex2(s[i][3] - g1);
                l0 += e0 + e1;
                l1 += e2 + e3;
                pa[i >> 1][(i & 1) * 2] = pack_h2(e0, e1);
                pa[i >> 1][(i & 1) * 2 + 1] = pack_h2(e2, e3);
            }
            const uint32_t v_base = smem_addr(Vs + (st * KT + (lane & 15)) * LV + (lane >> 4) * 8);
#pragma unroll
            for (int j = 0; j < KT / 16; j++) {
#pragma unroll
                for (int i = 0; i < DV / 8; i += 2) {
                    if (i * 8 < dv) {
                        uint32_t b[4];
                        ldsm4_t(v_base + (j * 16 * LV + i * 8) * 2, b);
                        mma_f16(o[i], pa[j], b[0], b[1]);
                        mma_f16(o[i + 1], pa[j], b[2], b[3]);
                    }
                }
            }
        }
        __syncthreads();                                // this stage may be refilled
    }
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    if (a.sink) { l0 += exp2f(sink - m0); l1 += exp2f(sink - m1); }
    float i0 = l0 > 0.f ? out_scale(a) / l0 : 0.f, i1 = l1 > 0.f ? out_scale(a) / l1 : 0.f;
    if (a.gate_col >= 0 && !a.gate_wide) {
        if (r0 < n) i0 *= sigmoidf(qkv[(size_t)(tl.x + r0) * ld + a.gate_col + h]);
        if (r1 < n) i1 *= sigmoidf(qkv[(size_t)(tl.x + r1) * ld + a.gate_col + h]);
    }
    const bool pairs = (a.vdim & 1) == 0 && (out_ld & 1) == 0;
#pragma unroll
    for (int i = 0; i < DV / 8; i++) {
        const int d = i * 8 + 2 * t;
        if (a.gate_wide && d < a.vdim) {
            const float* g0 = qkv + (size_t)(tl.x + r0) * ld + a.gate_col + h * a.vdim + d;
            const float* g1 = g0 + (size_t)8 * ld;
            if (r0 < n) { o[i][0] *= sigmoidf(g0[0]); if (d + 1 < a.vdim) o[i][1] *= sigmoidf(g0[1]); }
            if (r1 < n) { o[i][2] *= sigmoidf(g1[0]); if (d + 1 < a.vdim) o[i][3] *= sigmoidf(g1[1]); }
        }
        __nv_bfloat16* a0 = out + (size_t)(tl.x + r0) * out_ld + h * a.vdim + d;
        __nv_bfloat16* a1 = out + (size_t)(tl.x + r1) * out_ld + h * a.vdim + d;
        if (pairs) {
            if (d < a.vdim) {
                if (r0 < n) *reinterpret_cast<__nv_bfloat162*>(a0) = __floats2bfloat162_rn(o[i][0] * i0, o[i][1] * i0);
                if (r1 < n) *reinterpret_cast<__nv_bfloat162*>(a1) = __floats2bfloat162_rn(o[i][2] * i1, o[i][3] * i1);
            }
        } else {
            if (d < a.vdim) {
                if (r0 < n) a0[0] = __float2bfloat16_rn(o[i][0] * i0);
                if (r1 < n) a1[0] = __float2bfloat16_rn(o[i][2] * i1);
            }
            if (d + 1 < a.vdim) {
                if (r0 < n) a0[1] = __float2bfloat16_rn(o[i][1] * i0);
                if (r1 < n) a1[1] = __float2bfloat16_rn(o[i][3] * i1);
            }
        }
    }
}

constexpr int ONE_THREADS = 128, ONE_WARPS = ONE_THREADS / 32;

// grid = (splits, kv_heads * passes, rows), clusters of `splits` CTAs along x. Pass b of a key/value
// head serves its query heads b * RM .. b * RM + RM - 1. A lane owns VP * 2 consecutive value columns. SCORED: scores come from
// a.scores, the row's own among them, and the cache holds the row's value already.
template <int RM, int VP, bool SCORED>
__global__ void __launch_bounds__(ONE_THREADS)
attention_one_kernel(const cmlb200_attn a, const float* __restrict__ qkv, int ld, const int* __restrict__ row_pos, const int* __restrict__ row_slot,
                     __nv_bfloat16* __restrict__ out, int out_ld) {
    extern __shared__ __align__(16) float fs[];
    const int dk = a.dim_ld, dv = a.vdim_ld, group = a.heads / a.kv_heads, passes = (group + RM - 1) / RM;
    float* q_s = fs;                                   // [RM][dk], normed, rotated and scaled
    float* k_new = q_s + (SCORED ? 0 : RM * dk);       // [dk] and [dv] as the cache holds them
    float* v_new = k_new + (SCORED ? 0 : dk);
    float* turn = v_new + (SCORED ? 0 : dv);           // [rot_dims]: cosines, then sines
    float* w_m = turn + (SCORED || !a.freq ? 0 : a.rot_dims);                         // [ONE_WARPS][RM] maxima and sums
    float* w_l = w_m + ONE_WARPS * RM;
    float* c_m = w_l + ONE_WARPS * RM;                 // [RM] this CTA's
    float* c_l = c_m + RM;
    float* w_acc = c_l + RM;                           // [ONE_WARPS][RM][dv]; the CTA's sums end up in warp 0's part
    __shared__ float2 red[ONE_WARPS];
    dep_wait();
    dep_trigger();
    const int splits = gridDim.x, rank = blockIdx.x, kh = blockIdx.y / passes, pass = blockIdx.y % passes, r = blockIdx.z;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int h0 = kh * group + pass * RM, nh = min(RM, group - pass * RM);
    const float* row = qkv + (size_t)r * ld;
    const int p = row_pos[r], qw = a.heads * a.dim, kw = a.kv_heads * a.dim;
    const int shift = __ffs(a.block_size) - 1;
    const int* table = a.block_table + (size_t)row_slot[r] * a.table_ld;

    if constexpr (!SCORED) {
        float iq = 1.0f, ik = 1.0f;
        __shared__ float head_inv[RM + 1];             // per-head norms: of this CTA's query heads, then of its key
        if (a.freq) {
            const int half = a.rot_dims / 2;
            for (int i = threadIdx.x; i < half; i += ONE_THREADS) sincosf((float)p * a.freq[i], &turn[half + i], &turn[i]);
            __syncthreads();
        }
        if (a.head_norm) {
            for (int j = warp; j <= nh; j += ONE_WARPS) {
                const float* v = j < nh ? row + (h0 + j) * a.dim : row + qw + kh * a.dim;
                float ss = 0.f;
                for (int d = lane; d < a.dim; d += 32) ss = fmaf(v[d], v[d], ss);
                ss = lane_sum(ss);
                if (lane == 0) head_inv[j < nh ? j : RM] = (j < nh ? a.q_norm : a.k_norm) ? 1.0f / sqrtf(ss / (float)a.dim + a.eps) : 1.0f;
            }
            __syncthreads();
        } else if (a.q_norm || a.k_norm) {
            const float2 ss = block_sum2(a.q_norm ? square_share(row, qw) : 0.f, a.k_norm && rank == 0 ? square_share(row + qw, kw) : 0.f, red);
            if (a.q_norm) iq = 1.0f / sqrtf(ss.x / (float)qw + a.eps);
            if (a.k_norm) ik = 1.0f / sqrtf(ss.y / (float)kw + a.eps);  // used where the row's own key is made: rank 0
        }
        const float temp = a.temp_every > 0.f ? 1.0f + a.temp_coef * logf(floorf((float)(p + 1) / a.temp_every) + 1.0f) : 1.0f;
        const float qs = a.scale * kLog2e;
        // entry d of a head's vector v, turned with the one beside it
        auto turned = [&](int d, auto v) {
            if (!a.freq || d >= a.rot_dims) return v(d);
            const float c = turn[d >> 1], n = turn[(a.rot_dims + d) >> 1];
            return (d & 1) ? v(d) * c + v(d - 1) * n : v(d) * c - v(d + 1) * n;
        };
        for (int i = threadIdx.x; i < RM * dk; i += ONE_THREADS) {
            const int j = i / dk, d0 = i - j * dk;
            q_s[i] = (j < nh && d0 < a.dim) ? turned(d0, [&](int d) {
                const int c = (h0 + j) * a.dim + d;
                return row[c] * (a.head_norm ? head_inv[j] : iq) * (a.q_norm ? a.q_norm[a.head_norm ? d : c] : 1.0f) * temp * qs;
            }) : 0.f;
        }
        if (rank == 0) {
            const size_t slot = ((size_t)table[p >> shift] << shift) + (p & (a.block_size - 1));
            __half* kd = static_cast<__half*>(a.k_pool) + (slot * a.kv_heads + kh) * dk;
            __half* vd = static_cast<__half*>(a.v_pool) + (slot * a.kv_heads + kh) * dv;
            for (int d0 = threadIdx.x; d0 < dk; d0 += ONE_THREADS) {
                const __half v = narrow<__half>(d0 < a.dim ? turned(d0, [&](int d) {
                    const int c = kh * a.dim + d;
                    return row[qw + c] * (a.head_norm ? head_inv[RM] : ik) * (a.k_norm ? a.k_norm[a.head_norm ? d : c] : 1.0f);
                }) : 0.f);
                k_new[d0] = __half2float(v);
                if (pass == 0) kd[d0] = v;
            }
            for (int d = threadIdx.x; d < dv; d += ONE_THREADS) {
                const __half v = narrow<__half>(d < a.vdim ? row[qw + (a.keys_as_values ? 0 : kw) + kh * a.vdim + d] : 0.f);
                v_new[d] = __half2float(v);
                if (pass == 0) vd[d] = v;
            }
        }
        __syncthreads();
    }

    float m[RM], l[RM], acc[RM][2 * VP], slope[RM];
#pragma unroll
    for (int j = 0; j < RM; j++) {
        m[j] = -INFINITY;
        l[j] = 0.f;
        slope[j] = (a.slopes && j < nh) ? a.slopes[h0 + j] * kLog2e : 0.f;
#pragma unroll
        for (int e = 0; e < 2 * VP; e++) acc[j][e] = 0.f;
    }
    // the keys in sight, numbered from 0: the kept ones, then those from k_lo on
    const int k_lo = first_key(a, p), kept = min(a.keep, k_lo), skip = k_lo - kept, seen = p - skip + (SCORED ? 1 : 0);
    const __half* kp = static_cast<const __half*>(a.k_pool) + (size_t)kh * dk;
    const __half* vp = static_cast<const __half*>(a.v_pool) + (size_t)kh * dv;
    const int kstride = a.kv_heads * dk, vstride = a.kv_heads * dv;
    const int vcol = lane * 2 * VP;
    const bool has_v = vcol < dv;
    constexpr int PRE = VP == 4 ? 8 : 16;
    auto load_values = [&](uint32_t (&u)[PRE][VP], int slot, int k0) {
#pragma unroll
        for (int k = 0; k < PRE; k++) {
            const int ks = __shfl_sync(0xffffffffu, slot, k0 + k);       // lanes past the last key hold its slot
#pragma unroll
            for (int e = 0; e < VP; e++) u[k][e] = 0u;
            if (!has_v) continue;
            const __half* src = vp + (size_t)ks * vstride + vcol;
            if (VP == 4) { const uint4 w = *reinterpret_cast<const uint4*>(src); u[k][0] = w.x; u[k][1 % VP] = w.y; u[k][2 % VP] = w.z; u[k][3 % VP] = w.w; }
            else if (VP == 2) { const uint2 w = *reinterpret_cast<const uint2*>(src); u[k][0] = w.x; u[k][1 % VP] = w.y; }
            else u[k][0] = *reinterpret_cast<const uint32_t*>(src);
        }
    };
    // cached keys, 32 per warp and step; a lane scores one key
    for (int kt = (rank * ONE_WARPS + warp) * 32; kt < seen; kt += splits * ONE_WARPS * 32) {
        const int count = min(32, seen - kt), nth = min(kt + lane, seen - 1);
        const int key = nth + (nth < kept ? 0 : skip), kc = key;
        const int slot = (table[kc >> shift] << shift) + (kc & (a.block_size - 1));
        float s[RM];
#pragma unroll
        for (int j = 0; j < RM; j++) s[j] = 0.f;
        // the value rows do not depend on the scores: the first PRE of them are requested ahead of the keys
        uint32_t u[PRE][VP];
        load_values(u, slot, 0);
        const uint4* kr = reinterpret_cast<const uint4*>(kp + (size_t)slot * kstride);
        if constexpr (SCORED) {
#pragma unroll
            for (int j = 0; j < RM; j++) s[j] = a.scores[((size_t)r * a.heads + h0 + min(j, nh - 1)) * a.scores_ld + nth];
        }
#pragma unroll 8
        for (int c = 0; c < (SCORED ? 0 : dk >> 3); c++) {
            const uint4 w = kr[c];
            const float2 k01 = __half22float2(*reinterpret_cast<const __half2*>(&w.x)), k23 = __half22float2(*reinterpret_cast<const __half2*>(&w.y));
            const float2 k45 = __half22float2(*reinterpret_cast<const __half2*>(&w.z)), k67 = __half22float2(*reinterpret_cast<const __half2*>(&w.w));
#pragma unroll
            for (int j = 0; j < RM; j++) {
                const float4 x = *reinterpret_cast<const float4*>(q_s + j * dk + c * 8), y = *reinterpret_cast<const float4*>(q_s + j * dk + c * 8 + 4);
                s[j] = fmaf(x.x, k01.x, fmaf(x.y, k01.y, fmaf(x.z, k23.x, fmaf(x.w, k23.y, s[j]))));
                s[j] = fmaf(y.x, k45.x, fmaf(y.y, k45.y, fmaf(y.z, k67.x, fmaf(y.w, k67.y, s[j]))));
            }
        }
#pragma unroll
        for (int j = 0; j < RM; j++) {
            const float v = lane < count ? s[j] - slope[j] * (float)(p - key) : -INFINITY;
            const float mn = fmaxf(m[j], lane_max(v));
            const float c = exp2f(m[j] - mn);
            m[j] = mn;
            s[j] = exp2f(v - mn);
            l[j] = l[j] * c + s[j];
#pragma unroll
            for (int e = 0; e < 2 * VP; e++) acc[j][e] *= c;
        }
        for (int k0 = 0; k0 < count; k0 += PRE) {
            if (k0) load_values(u, slot, k0);
#pragma unroll
            for (int k = 0; k < PRE; k++) {            // weights past the last key are zero
#pragma unroll
                for (int j = 0; j < RM; j++) {
                    const float w = __shfl_sync(0xffffffffu, s[j], k0 + k);
#pragma unroll
                    for (int e = 0; e < VP; e++) {
                        const float2 v = __half22float2(*reinterpret_cast<const __half2*>(&u[k][e]));
                        acc[j][2 * e] = fmaf(w, v.x, acc[j][2 * e]);
                        acc[j][2 * e + 1] = fmaf(w, v.y, acc[j][2 * e + 1]);
                    }
                }
            }
        }
    }
#pragma unroll
    for (int j = 0; j < RM; j++) l[j] = lane_sum(l[j]);
    if (!SCORED && rank == 0 && warp == 0) {           // the row's own key and value, distance 0
#pragma unroll
        for (int j = 0; j < RM; j++) {
            float s = 0.f;
            for (int d = lane; d < dk; d += 32) s = fmaf(q_s[j * dk + d], k_new[d], s);
            s = lane_sum(s);
            const float mn = fmaxf(m[j], s), c = exp2f(m[j] - mn), w = exp2f(s - mn);
            m[j] = mn;
            l[j] = l[j] * c + w;
#pragma unroll
            for (int e = 0; e < 2 * VP; e++) acc[j][e] = acc[j][e] * c + (has_v ? w * v_new[vcol + e] : 0.f);
        }
    }
    // ---- merge the warps, then the CTAs of the cluster
#pragma unroll
    for (int j = 0; j < RM; j++) {
        if (lane == 0) { w_m[warp * RM + j] = m[j]; w_l[warp * RM + j] = l[j]; }
        if (has_v)
#pragma unroll
            for (int e = 0; e < 2 * VP; e++) w_acc[(warp * RM + j) * dv + vcol + e] = acc[j][e];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < RM * dv; i += ONE_THREADS) {
        const int j = i / dv;
        float mx = w_m[j];
#pragma unroll
        for (int w = 1; w < ONE_WARPS; w++) mx = fmaxf(mx, w_m[w * RM + j]);
        float x = 0.f, sum = 0.f;
#pragma unroll
        for (int w = 0; w < ONE_WARPS; w++) {
            const float mw = w_m[w * RM + j], c = mw == -INFINITY ? 0.f : exp2f(mw - mx);
            x = fmaf(w_acc[w * RM * dv + i], c, x);
            sum = fmaf(w_l[w * RM + j], c, sum);
        }
        w_acc[i] = x;                                  // element i of warp 0's part is read and written by this thread alone
        if (i - j * dv == 0) { c_m[j] = mx; c_l[j] = sum; }
    }
    if (splits > 1) {
        asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
        asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    } else {
        __syncthreads();
    }
    if (rank == 0) {
        for (int i = threadIdx.x; i < nh * dv; i += ONE_THREADS) {
            const int j = i / dv, d = i - j * dv;
            float x, sum, mx;
            if (splits > 1) {
                float ms[8], ls[8], xs[8];
#pragma unroll
                for (int s = 0; s < 8; s++) {
                    ms[s] = -INFINITY; ls[s] = 0.f; xs[s] = 0.f;
                    if (s < splits) {
                        uint32_t am, al, ax;
                        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(am) : "r"(smem_addr(c_m + j)), "r"(s));
                        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(al) : "r"(smem_addr(c_l + j)), "r"(s));
                        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(ax) : "r"(smem_addr(w_acc + i)), "r"(s));
                        asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(ms[s]) : "r"(am) : "memory");
                        asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(ls[s]) : "r"(al) : "memory");
                        asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(xs[s]) : "r"(ax) : "memory");
                    }
                }
                mx = ms[0];
#pragma unroll
                for (int s = 1; s < 8; s++) mx = fmaxf(mx, ms[s]);
                x = 0.f; sum = 0.f;
#pragma unroll
                for (int s = 0; s < 8; s++) {
                    const float c = ms[s] == -INFINITY ? 0.f : exp2f(ms[s] - mx);
                    x = fmaf(xs[s], c, x);
                    sum = fmaf(ls[s], c, sum);
                }
            } else {
                x = w_acc[i]; sum = c_l[j]; mx = c_m[j];
            }
            if (a.sink) {                              // it carries no value
                const float sk = sink_score(a, h0 + j) * kLog2e, mt = fmaxf(mx, sk), c = exp2f(mx - mt);
                x *= c;
                sum = sum * c + exp2f(sk - mt);
            }
            float v = x / sum * out_scale(a);
            if (a.gate_col >= 0) v *= sigmoidf(row[a.gate_col + h0 + j]);
            if (d < a.vdim) out[(size_t)r * out_ld + (h0 + j) * a.vdim + d] = __float2bfloat16_rn(v);
        }
    }
    if (splits > 1) {                                  // nobody leaves while rank 0 reads its shared memory
        asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
        asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    }
}

constexpr int ROW_THREADS = 128;

// grid = (rows, heads); q already normed (in place in the projection rows). Keys in chunks of 128:
// a warp scores a key at a time, the running maximum and sum are per CTA.
__global__ void __launch_bounds__(ROW_THREADS)
attention_rows_f32_kernel(const cmlb200_attn a, const float* __restrict__ qkv, int ld, const int* __restrict__ row_pos,
                          const int* __restrict__ row_slot, float* __restrict__ out, int out_ld) {
    extern __shared__ __align__(16) float fs[];
    float* q_s = fs;                                   // [dim]
    float* acc = q_s + a.dim;                          // [vdim]
    __shared__ float sc[ROW_THREADS], red[32];
    __shared__ int slots[ROW_THREADS];
    dep_wait();
    dep_trigger();
    const int r = blockIdx.x, h = blockIdx.y, kh = h / (a.heads / a.kv_heads), lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const float* row = qkv + (size_t)r * ld;
    const int p = row_pos[r];
    const int* table = a.block_table + (size_t)row_slot[r] * a.table_ld;
    const float* kp = static_cast<const float*>(a.k_pool) + (size_t)kh * a.dim_ld;
    const float* vp = static_cast<const float*>(a.v_pool) + (size_t)kh * a.vdim_ld;
    const float slope = a.slopes ? a.slopes[h] : 0.f;
    const float* given = a.scores ? a.scores + ((size_t)r * a.heads + h) * a.scores_ld : nullptr;
    for (int d = threadIdx.x; d < a.dim && !given; d += ROW_THREADS) q_s[d] = row[h * a.dim + d];
    for (int d = threadIdx.x; d < a.vdim; d += ROW_THREADS) acc[d] = 0.f;
    float m = a.sink ? sink_score(a, h) : -INFINITY, l = a.sink ? 1.f : 0.f;
    const int k_lo = first_key(a, p), kept = min(a.keep, k_lo), skip = k_lo - kept, seen = p + 1 - skip;
    auto key_of = [&](int nth) { return nth + (nth < kept ? 0 : skip); };
    for (int kt = 0; kt < seen; kt += ROW_THREADS) {
        const int n = min(ROW_THREADS, seen - kt);
        __syncthreads();                               // the previous chunk's weights are consumed (and q_s is there)
        if ((int)threadIdx.x < n) {
            const int key = key_of(kt + threadIdx.x);
            slots[threadIdx.x] = table[key / a.block_size] * a.block_size + key % a.block_size;
        }
        __syncthreads();
        if (given && (int)threadIdx.x < n) sc[threadIdx.x] = given[kt + threadIdx.x];
        for (int k = warp; k < n && !given; k += ROW_THREADS / 32) {
            const float* kr = kp + (size_t)slots[k] * a.kv_heads * a.dim_ld;
            float s = 0.f;
            for (int d = lane; d < a.dim; d += 32) s = fmaf(q_s[d], kr[d], s);
            s = lane_sum(s);
            if (lane == 0) sc[k] = s * a.scale - slope * (float)(p - key_of(kt + k));
        }
        __syncthreads();
        float mx = m;
        for (int k = 0; k < n; k++) mx = fmaxf(mx, sc[k]);
        const float c = expf(m - mx);
        m = mx;
        const float w = (int)threadIdx.x < n ? expf(sc[threadIdx.x] - mx) : 0.f;
        l = l * c + block_sum(w, red);                 // the barriers inside also order the reads of sc above
        sc[threadIdx.x] = w;
        __syncthreads();
        for (int d = threadIdx.x; d < a.vdim; d += ROW_THREADS) {
            float x = acc[d] * c;
            for (int k = 0; k < n; k++) x = fmaf(sc[k], vp[(size_t)slots[k] * a.kv_heads * a.vdim_ld + d], x);
            acc[d] = x;
        }
    }
    const float inv = (a.gate_col >= 0 ? sigmoidf(row[a.gate_col + h]) : 1.0f) * out_scale(a) / l;
    for (int d = threadIdx.x; d < a.vdim; d += ROW_THREADS) out[(size_t)r * out_ld + h * a.vdim + d] = acc[d] * inv;
}

}  // namespace

// Shape and alignment checks shared by the entry points that take a cmlb200_attn.
extern "C" int cmlb200_attn_check_(const cmlb200_attn* a, const char* who) {
    CMLB_REQUIRE(a->heads > 0 && a->kv_heads > 0 && a->heads % a->kv_heads == 0, "%s: heads %d, kv_heads %d", who, a->heads, a->kv_heads);
    CMLB_REQUIRE(a->dim > 0 && a->vdim > 0 && a->dim_ld >= a->dim && a->vdim_ld >= a->vdim && a->dim_ld % 16 == 0 && a->vdim_ld % 16 == 0,
                 "%s: head sizes %d (stride %d) / %d (stride %d)", who, a->dim, a->dim_ld, a->vdim, a->vdim_ld);
    CMLB_REQUIRE(a->cache_dtype == CMLB200_DT_F32 || a->cache_dtype == CMLB200_DT_F16, "%s: cache dtype %d", who, a->cache_dtype);
    CMLB_REQUIRE(!a->gate_wide || a->gate_col >= 0, "%s: gate_wide without a gate column", who);
    CMLB_REQUIRE(a->keep >= 0 && a->chunk >= 0 && (!a->keys_as_values || a->dim == a->vdim), "%s: kept tokens %d, chunk %d, values as keys of %d / %d", who, a->keep,
                 a->chunk, a->dim, a->vdim);
    CMLB_REQUIRE(a->k_pool && a->v_pool && a->block_table && a->table_ld > 0, "%s: no cache", who);
    CMLB_REQUIRE(!a->scores || (a->scores_ld > 0 && !a->slopes && a->chunk == 0 && a->keep == 0), "%s: given scores go with windows alone, stride %d", who, a->scores_ld);
    CMLB_REQUIRE(!a->freq || (a->rot_dims > 0 && a->rot_dims % 2 == 0 && a->rot_dims <= a->dim), "%s: %d of %d dimensions rotated", who, a->rot_dims, a->dim);
    CMLB_REQUIRE(a->block_size > 0 && (a->block_size & (a->block_size - 1)) == 0 && a->block_size % 16 == 0, "%s: block size %d must be a power of two >= 16", who, a->block_size);
    CMLB_REQUIRE((((uintptr_t)a->k_pool | (uintptr_t)a->v_pool) & 15) == 0, "%s: pools must be 16-byte aligned", who);
    return CMLB200_OK;
}

extern "C" int cmlb200_attention_tiles(const cmlb200_attn* a, const float* d_qkv, int ld, const int* d_tiles, int tiles, uint16_t* d_out_bf16,
                                       int out_ld, void* stream) {
    CMLB_REQUIRE(a && d_qkv && d_tiles && tiles > 0 && d_out_bf16, "cmlb200_attention_tiles: bad argument");
    const int rc = cmlb200_attn_check_(a, "cmlb200_attention_tiles");
    if (rc) return rc;
    CMLB_REQUIRE(a->cache_dtype == CMLB200_DT_F16 && a->vdim_ld <= 256 && a->heads <= 65535, "cmlb200_attention_tiles: fp16 cache and value heads up to 256");
    CMLB_REQUIRE(((uintptr_t)d_tiles & 15) == 0, "cmlb200_attention_tiles: the tile list must be 16-byte aligned");
    const bool scored = a->scores != nullptr;
    CMLB_REQUIRE(!scored || (a->scores_ld % 64 == 0 && ((uintptr_t)a->scores & 15) == 0), "cmlb200_attention_tiles: score stride %d", a->scores_ld);
    const size_t smem = 2 * ((scored ? 0 : (size_t)(QT + 2 * KT) * (a->dim_ld + 8)) + (size_t)2 * KT * (a->vdim_ld + 8));
    CMLB_REQUIRE(smem <= 227 * 1024, "cmlb200_attention_tiles: head sizes %d / %d do not fit shared memory", a->dim, a->vdim);
    cudaStream_t st = as_stream(stream);
    const dim3 grid(tiles, a->heads);
    static size_t attr[9][kMaxDevices] = {};
#define AT_LAUNCH(DV, DK, S, slot)                                                                                                   \
    do {                                                                                                                        \
        auto kern = attention_tiles_kernel<DV, DK, S>;                                                                               \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                    \
        CMLB_CUDA(launch_chain(kern, grid, dim3(TILE_THREADS), smem, 1, st, *a, d_qkv, ld, (const int4*)d_tiles, (__nv_bfloat16*)d_out_bf16, out_ld)); \
    } while (0)
    if (scored) {
        if (a->vdim_ld <= 64) AT_LAUNCH(64, 0, true, 6);
        else if (a->vdim_ld <= 128) AT_LAUNCH(128, 0, true, 7);
        else AT_LAUNCH(256, 0, true, 8);
    }
    else if (a->vdim_ld == 64 && a->dim_ld == 64) AT_LAUNCH(64, 64, false, 3);
    else if (a->vdim_ld == 128 && a->dim_ld == 128) AT_LAUNCH(128, 128, false, 4);
    else if (a->vdim_ld == 128 && a->dim_ld == 192) AT_LAUNCH(128, 192, false, 5);
    else if (a->vdim_ld <= 64) AT_LAUNCH(64, 0, false, 0);
    else if (a->vdim_ld <= 128) AT_LAUNCH(128, 0, false, 1);
    else AT_LAUNCH(256, 0, false, 2);
#undef AT_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_attention_one(const cmlb200_attn* a, const float* d_qkv, int ld, const int* d_row_pos, const int* d_row_slot, int rows,
                                     int max_keys, uint16_t* d_out_bf16, int out_ld, void* stream) {
    CMLB_REQUIRE(a && d_qkv && d_row_pos && d_row_slot && rows > 0 && max_keys >= 0 && d_out_bf16, "cmlb200_attention_one: bad argument");
    const int rc = cmlb200_attn_check_(a, "cmlb200_attention_one");
    if (rc) return rc;
    CMLB_REQUIRE(a->cache_dtype == CMLB200_DT_F16 && a->vdim_ld <= 256 && rows <= 65535, "cmlb200_attention_one: fp16 cache and value heads up to 256");
    CMLB_REQUIRE(!a->gate_wide, "cmlb200_attention_one: one gate per head");
    // few rows: fewer heads per CTA, so that more CTAs share the work (the keys are read again from L2)
    const int group = a->heads / a->kv_heads, rm = group == 1 ? 1 : (group <= 4 || rows * a->kv_heads * 8 < cmlb_num_sms() ? 4 : 8), passes = (group + rm - 1) / rm;
    CMLB_REQUIRE((long long)a->kv_heads * passes <= 65535, "cmlb200_attention_one: too many heads");
    const int reach = a->chunk > 0 ? a->chunk : a->window;
    const int keys = (reach > 0 && reach < max_keys - a->keep) ? reach + a->keep : max_keys;
    const long long base = (long long)rows * a->kv_heads * passes;
    int splits = 1;
    while (splits < 8 && base * splits < 2 * cmlb_num_sms() && keys > splits * ONE_WARPS * 32) splits *= 2;
    const bool scored = a->scores != nullptr;
    CMLB_REQUIRE(!scored || a->scores_ld >= keys, "cmlb200_attention_one: score stride %d for %d keys", a->scores_ld, keys);
    const size_t operands = scored ? 0 : (size_t)rm * a->dim_ld + a->dim_ld + a->vdim_ld + (a->freq ? a->rot_dims : 0);
    const size_t smem = sizeof(float) * (operands + 2 * ONE_WARPS * rm + 2 * rm + (size_t)ONE_WARPS * rm * a->vdim_ld);
    CMLB_REQUIRE(smem <= 200 * 1024, "cmlb200_attention_one: head sizes %d / %d do not fit shared memory", a->dim, a->vdim);
    cudaStream_t st = as_stream(stream);
    const dim3 grid(splits, a->kv_heads * passes, rows);
    const int vp = a->vdim_ld <= 64 ? 1 : (a->vdim_ld <= 128 ? 2 : 4);
    static size_t attr[18][kMaxDevices] = {};
#define AO_LAUNCH(RM, VP, S, slot)                                                                                                  \
    do {                                                                                                                         \
        auto kern = attention_one_kernel<RM, VP, S>;                                                                                \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                     \
        CMLB_CUDA(launch_chain(kern, grid, dim3(ONE_THREADS), smem, splits, st, *a, d_qkv, ld, d_row_pos, d_row_slot, (__nv_bfloat16*)d_out_bf16, out_ld)); \
    } while (0)
#define AO_ROWS(RM, S, slot)                                \
    do {                                                    \
        if (vp == 1) AO_LAUNCH(RM, 1, S, slot);             \
        else if (vp == 2) AO_LAUNCH(RM, 2, S, slot + 1);    \
        else AO_LAUNCH(RM, 4, S, slot + 2);                 \
    } while (0)
#define AO_FORM(S, slot)                                    \
    do {                                                    \
        if (rm == 1) AO_ROWS(1, S, slot);                   \
        else if (rm == 4) AO_ROWS(4, S, slot + 3);          \
        else AO_ROWS(8, S, slot + 6);                       \
    } while (0)
    if (scored) AO_FORM(true, 9);
    else AO_FORM(false, 0);
#undef AO_FORM
#undef AO_ROWS
#undef AO_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_attention_rows_f32(const cmlb200_attn* a, const float* d_qkv, int ld, const int* d_row_pos, const int* d_row_slot, int rows,
                                          float* d_out, int out_ld, void* stream) {
    CMLB_REQUIRE(a && d_qkv && d_row_pos && d_row_slot && rows > 0 && d_out, "cmlb200_attention_rows_f32: bad argument");
    const int rc = cmlb200_attn_check_(a, "cmlb200_attention_rows_f32");
    if (rc) return rc;
    CMLB_REQUIRE(a->cache_dtype == CMLB200_DT_F32 && a->heads <= 65535, "cmlb200_attention_rows_f32: fp32 cache");
    CMLB_REQUIRE(!a->gate_wide, "cmlb200_attention_rows_f32: one gate per head");
    const size_t smem = sizeof(float) * ((size_t)a->dim + a->vdim);
    CMLB_REQUIRE(smem <= 40 * 1024, "cmlb200_attention_rows_f32: head sizes %d / %d", a->dim, a->vdim);
    CMLB_CUDA(launch_chain(attention_rows_f32_kernel, dim3(rows, a->heads), dim3(ROW_THREADS), smem, 1, as_stream(stream), *a, d_qkv, ld, d_row_pos,
                           d_row_slot, d_out, out_ld));
    return CMLB200_OK;
}
