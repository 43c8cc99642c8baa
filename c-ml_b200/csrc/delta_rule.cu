// Gated delta rule (see cmlb200_delta): a recurrence over tokens with one matrix of state per head, everything in fp32.
// With S read after the decay, s_k = S^T k and s_q = S^T q are sums over the same elements, and
//   u = beta (v - s_k),  o = s_q + (k . q) u,  S <- S + k u^T,
// so that a token needs one pass over S for both sums and one for the update.
//
//   delta_one_kernel      decoded tokens, one row per sequence: convolution, unit norms, decay, state, output norm and gate
//                         in one launch. A head's columns may be split over a cluster, which shares the output's square sum
//   delta_prepare_kernel  portions, cut into chunks of eight tokens: everything of a chunk that does not depend on the state, a
//                         warp per chunk and head
//   delta_scan_kernel     portions: the recurrence, a chunk at a time, on the tensor cores. A CTA keeps 16 columns of a
//                         head's state as accumulators, its warps a share of the key channels each
//   delta_output_kernel   portions: output norm and gate, a warp per (row, head)
//
// A chunk of eight tokens, G_i the product of the decays up to token i, G_ij of those after j up to i (all products of
// factors below one, nothing is ever divided by a decay): the sums over the state before the chunk are R_i = (k_i G_i)^T S
// and (q_i G_i)^T S, and with A_ij = (k_i G_ij) . k_j, B_ij = (q_i G_ij) . k_j (B_ii = q_i . k_i)
//   u_i = beta_i (v_i - R_i - sum_j<i A_ij u_j)  =  M (v - R),   M = (1 + beta A)^-1 beta,
//   o_i = (q_i G_i)^T S + sum_j<=i B_ij u_j,   S <- G_8 S + sum_j (k_j G_8j) u_j^T.
// Every product of matrices is fp32 to rounding: operands are split into two tf32 parts, and three products of the parts
// are added in fp32. Accumulators of one product have the layout of the next one's left operand when the columns of
// both operands are taken in the order 0 2 4 6 1 3 5 7, so nothing moves between lanes.
//
// A sequence's latest projections lie in a ring of `taps` entries, position p in entry p mod taps: a token reads the
// entries before its own and writes its own, so the heads that share a key may do both in any order.
#include "lm_util.cuh"

namespace {

constexpr float kUnitEps = 1e-6f;

__device__ __forceinline__ int delta_channels(const cmlb200_delta& a) { return 2 * a.kv_heads * a.dim + a.heads * a.vdim; }
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
// log(1 + e^z) = max(z, 0) + 2 artanh(e / (2 + e)) with e = e^-|z|: the argument of the series is at most 1/3, and nothing
// cancels where e is small.
__device__ __forceinline__ float softplus(float z) {
    const float e = __expf(-fabsf(z)), s = __fdividef(e, 2.0f + e), w = s * s;
    float p = 1.0f / 15.0f;
    p = fmaf(p, w, 1.0f / 13.0f);
    p = fmaf(p, w, 1.0f / 11.0f);
    p = fmaf(p, w, 1.0f / 9.0f);
    p = fmaf(p, w, 1.0f / 7.0f);
    p = fmaf(p, w, 1.0f / 5.0f);
    p = fmaf(p, w, 1.0f / 3.0f);
    p = fmaf(p, w, 1.0f);
    return fmaf(2.0f * s, p, fmaxf(z, 0.f));
}
__device__ __forceinline__ float decay(float rate, float z) { return expf(-rate * softplus(z)); }
__device__ __forceinline__ float delta_scale(const cmlb200_delta& a) { return a.out_scale == 0.f ? 1.f : a.out_scale; }

// Channel c at a decoded token's row: its own projection and those of the tokens before it, from the ring. T: the number of taps
// where it is known (all loads are then under way together), 0: any.
template <int T>
__device__ __forceinline__ float convolve(const cmlb200_delta& a, const float* __restrict__ proj, const float* __restrict__ ring, int channels, int c, int p) {
    const float now = proj[a.col + c];
    if constexpr (T > 0) {
        float w[T], x[T];
#pragma unroll
        for (int t = 0; t < T; t++) {
            w[t] = a.conv[(size_t)(T - 1 - t) * channels + c];
            x[t] = t == 0 ? now : (t <= p ? ring[(size_t)((p - t) % T) * channels + c] : 0.f);
        }
        float y = 0.f;
#pragma unroll
        for (int t = 0; t < T; t++) y = fmaf(w[t], x[t], y);
        return silu_fast(y);
    }
    float y = a.conv[(size_t)(a.taps - 1) * channels + c] * now;
    for (int t = 1; t < a.taps && t <= p; t++) y = fmaf(a.conv[(size_t)(a.taps - 1 - t) * channels + c], ring[(size_t)((p - t) % a.taps) * channels + c], y);
    return silu_fast(y);
}

constexpr int ONE_THREADS = 256, ONE_WARPS = ONE_THREADS / 32;

// grid = (splits, heads, rows), clusters of `splits` CTAs along x. Thread (rg, c): four columns 4c of every `groups`-th row
// from rg on; RPT: room for those rows. lanes: threads across the columns of a CTA, a power of two.
template <typename TO, int RPT, int T>
__global__ void __launch_bounds__(ONE_THREADS, RPT <= 4 ? 4 : (RPT <= 8 ? 3 : (RPT <= 16 ? 2 : 1)))
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
    // positions, slots and states do not come from the launch in front, so the states are under way while that one ends
    const int p = row_pos[r], slot = row_slot[r];
    float4* state = reinterpret_cast<float4*>(a.state + ((size_t)slot * a.heads + h) * a.dim * a.vdim_ld + c0);
    const bool mine = 4 * c < cols && c0 < a.vdim_ld;
    float4 S[RPT];
#pragma unroll
    for (int i = 0; i < RPT; i++) {
        const int d = rg + i * groups;
        S[i] = mine && p > 0 && d < a.dim ? state[(size_t)d * (a.vdim_ld >> 2)] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    dep_wait();
    dep_trigger();
    const float* row = proj + (size_t)r * ld;
    float* ring = a.ring + (size_t)slot * a.taps * channels;
    float sq = 0.f, sk = 0.f;
    const bool keeps = rank == 0 && h == kh * group;
    for (int i = tid; i < 2 * a.dim + cols; i += ONE_THREADS) {        // q, k and this CTA's values
        const int which = i < a.dim ? 0 : (i < 2 * a.dim ? 1 : 2), d = i - which * a.dim, col = rank * cols + d;
        const int ch = which == 2 ? 2 * a.kv_heads * a.dim + h * a.vdim + col : (which * a.kv_heads + kh) * a.dim + d;
        const bool have = which < 2 || col < a.vdim;
        const float y = have ? convolve<T>(a, row, ring, channels, ch, p) : 0.f;
        (which == 0 ? q_s : (which == 1 ? k_s : v_s))[d] = y;
        sq += which == 0 ? y * y : 0.f;
        sk += which == 1 ? y * y : 0.f;
        if (have && (keeps || which == 2)) ring[(size_t)(p % a.taps) * channels + ch] = row[a.col + ch];
    }
    for (int d = tid; d < a.dim; d += ONE_THREADS) g_s[d] = decay(a.rate[h], dec[(size_t)r * ld_dec + h * a.dim + d] + a.dt_bias[h * a.dim + d]);
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

// What the scan needs of a chunk and head: per 8 key channels (a tile) k G and q G as [token][k k q q, four times], k G_8 as
// [channel][token], G_8; then M and B as [token][token], and the factors that make k and q unit vectors, which none of the
// first three carry. tiles: 8-channel tiles, a size the scan is built for.
constexpr int CHUNK = 8;
__host__ __device__ inline int scan_tiles(const cmlb200_delta& a) { return a.dim <= 32 ? 4 : (a.dim <= 64 ? 8 : (a.dim <= 128 ? 16 : 32)); }
__host__ __device__ inline int packet_floats(int tiles) { return tiles * 200 + 144; }
__host__ __device__ inline int value_ld(const cmlb200_delta& a) { return (a.heads * a.vdim + 3) & ~3; }
// A run's first packet: runs do not overlap, and each has one packet more than its rows' share at most.
__device__ __forceinline__ int first_packet(const int4 run, int i, int first) { return (run.x - first) / CHUNK + i; }

// The sum over the warp of v[l] ends up on lane l.
__device__ __forceinline__ float scatter_sums(float (&v)[32]) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int n = 16; n > 0; n >>= 1) {
        const bool upper = lane & n;
#pragma unroll
        for (int i = 0; i < n; i++) {
            const float mine = upper ? v[n + i] : v[i], other = upper ? v[i] : v[n + i];
            v[i] = mine + __shfl_xor_sync(0xffffffffu, other, n);
        }
    }
    return v[0];
}

// grid = (packets, heads / 4). T: taps if known (all loads of a channel are then under way together), 0: any.
template <int T>
__global__ void __launch_bounds__(128, 3)
delta_prepare_kernel(const cmlb200_delta a, const float* __restrict__ proj, int ld, const float* __restrict__ dec, int ld_dec, const int* __restrict__ row_pos,
                     const int4* __restrict__ runs, int num_runs, int first, float* __restrict__ values, float* __restrict__ packets) {
    __shared__ float sums[4][96], betas[4][CHUNK];
    dep_wait();
    dep_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, h = blockIdx.y * 4 + warp;
    int at = -1, c0 = 0;                               // the run this packet belongs to, and the chunk's first token in it
    for (int i0 = 0; i0 < num_runs && at < 0; i0 += 32) {
        const int i = i0 + lane, c = i < num_runs ? (int)blockIdx.x - first_packet(runs[i], i, first) : -1;
        const unsigned hit = __ballot_sync(0xffffffffu, c >= 0 && c * CHUNK < (i < num_runs ? runs[i].y : 0));
        if (hit) { at = i0 + __ffs(hit) - 1; c0 = __shfl_sync(0xffffffffu, c, __ffs(hit) - 1) * CHUNK; }
    }
    if (at < 0 || h >= a.heads) return;
    const int4 run = runs[at];
    const int n = run.y, count = min(CHUNK, n - c0), p0 = row_pos[run.x], tiles = scan_tiles(a), channels = delta_channels(a);
    const int kh = h / (a.heads / a.kv_heads), kd = a.kv_heads * a.dim;
    const float* ring = a.ring + (size_t)run.z * a.taps * channels;
    const float* rows = proj + (size_t)run.x * ld + a.col;
    constexpr int PAST = T > 0 ? T - 1 : 0;
    static_assert(PAST <= CHUNK, "a chunk's history is the chunk before it or the ring");
    int off[CHUNK], past[PAST + 1];                    // of the rows that a chunk's convolutions read (past the end: the last), and of the tokens before it
    bool seen[PAST + 1];
#pragma unroll
    for (int j = 0; j < CHUNK; j++) off[j] = min(c0 + j, n - 1) * ld;
    const float* before = c0 > 0 ? rows : ring;
#pragma unroll
    for (int j = 0; j < PAST; j++) {
        const int t = c0 + j - PAST;
        seen[j] = p0 + t >= 0;
        past[j] = c0 > 0 ? t * ld : max(p0 + t, 0) % T * channels;
    }
    auto convolve_chunk = [&](int c, float (&y)[CHUNK]) {
#pragma unroll
        for (int j = 0; j < CHUNK; j++) y[j] = 0.f;
        if constexpr (T > 0) {
            float x[PAST + CHUNK];
#pragma unroll
            for (int j = 0; j < PAST; j++) x[j] = seen[j] ? before[past[j] + c] : 0.f;
#pragma unroll
            for (int j = 0; j < CHUNK; j++) x[PAST + j] = rows[off[j] + c];
#pragma unroll
            for (int t = 0; t < T; t++) {
                const float w = a.conv[(T - 1 - t) * channels + c];
#pragma unroll
                for (int j = 0; j < CHUNK; j++) y[j] = fmaf(w, x[j + T - 1 - t], y[j]);
            }
        } else {
            for (int t = 0; t < a.taps; t++) {
                const float w = a.conv[(a.taps - 1 - t) * channels + c];
#pragma unroll
                for (int j = 0; j < CHUNK; j++) {
                    const int at = c0 + j - t;         // a token of the run, or before it
                    const float x = at >= 0 ? rows[min(at, n - 1) * ld + c] : (p0 + at >= 0 ? ring[(p0 + at) % a.taps * channels + c] : 0.f);
                    y[j] = fmaf(w, x, y[j]);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < CHUNK; j++) y[j] = j < count ? silu_fast(y[j]) : 0.f;
    };
    float* packet = packets + ((size_t)blockIdx.x * a.heads + h) * packet_floats(tiles);
    float *kq = packet, *kt = kq + tiles * 128, *gt = kt + tiles * 64, *mat = gt + tiles * 8;
    float acc[96];                                     // A_ij, j < i, then B_ij, j <= i, then the square sums of q and of k
#pragma unroll
    for (int i = 0; i < 96; i++) acc[i] = 0.f;
    const float rate = a.rate[h];
    for (int d = lane; d < tiles * 8; d += 32) {
        float q[CHUNK], k[CHUNK], g[CHUNK], kg[CHUNK], qg[CHUNK], tail[CHUNK], run_g = 1.f;
        const bool have = d < a.dim;
        const int c = kh * a.dim + (have ? d : 0), gc = h * a.dim + (have ? d : 0);
        const float bias = a.dt_bias[gc];
#pragma unroll
        for (int j = 0; j < CHUNK; j++) g[j] = dec[(size_t)(run.x + min(c0 + j, n - 1)) * ld_dec + gc];
        convolve_chunk(c, q);
        convolve_chunk(kd + c, k);
#pragma unroll
        for (int j = 0; j < CHUNK; j++) {
            g[j] = j < count ? decay(rate, g[j] + bias) : 1.f;
            if (!have) { q[j] = 0.f; k[j] = 0.f; }
            run_g *= g[j];
            kg[j] = k[j] * run_g;
            qg[j] = q[j] * run_g;
            acc[64 + j] = fmaf(q[j], q[j], acc[64 + j]);
            acc[72 + j] = fmaf(k[j], k[j], acc[72 + j]);
        }
#pragma unroll
        for (int j = 0; j < CHUNK; j++) {
            float t = k[j];
            acc[28 + j * (j + 1) / 2 + j] = fmaf(q[j], t, acc[28 + j * (j + 1) / 2 + j]);
#pragma unroll
            for (int i = j + 1; i < CHUNK; i++) {
                t *= g[i];
                acc[i * (i - 1) / 2 + j] = fmaf(k[i], t, acc[i * (i - 1) / 2 + j]);
                acc[28 + i * (i + 1) / 2 + j] = fmaf(q[i], t, acc[28 + i * (i + 1) / 2 + j]);
            }
            tail[j] = t;
        }
        float* to = kq + (size_t)(d >> 3) * 128 + ((d & 7) >> 1) * 4 + (d & 1);
#pragma unroll
        for (int j = 0; j < CHUNK; j++) { to[j * 16] = kg[j]; to[j * 16 + 2] = qg[j]; }
        gt[d] = run_g;
        float4* end = reinterpret_cast<float4*>(kt + (size_t)d * CHUNK);
        end[0] = make_float4(tail[0], tail[1], tail[2], tail[3]);
        end[1] = make_float4(tail[4], tail[5], tail[6], tail[7]);
    }
#pragma unroll
    for (int b = 0; b < 3; b++) {
        float v[32];
#pragma unroll
        for (int i = 0; i < 32; i++) v[i] = acc[b * 32 + i];
        sums[warp][b * 32 + lane] = scatter_sums(v);
    }
    if (lane < CHUNK) betas[warp][lane] = lane < count ? sigmoidf(rows[(size_t)(c0 + lane) * ld + channels + h]) : 0.f;
    __syncwarp();
    float* sum = sums[warp];
    if (lane < CHUNK) {                                // from here on factors instead of square sums
        sum[64 + lane] = 1.0f / sqrtf(sum[64 + lane] + kUnitEps) / sqrtf((float)a.dim);
        sum[72 + lane] = 1.0f / sqrtf(sum[72 + lane] + kUnitEps);
        mat[136 + lane] = sum[64 + lane];
        mat[128 + lane] = sum[72 + lane];
    }
    __syncwarp();
    const float *iq = sum + 64, *ik = sum + 72;
    if (lane < CHUNK) {                                // a column of M by substitution
        float x[CHUNK];
#pragma unroll
        for (int i = 0; i < CHUNK; i++) {
            float s = 0.f;
#pragma unroll
            for (int j = 0; j < i; j++) s = fmaf(sum[i * (i - 1) / 2 + j] * ik[j], x[j], s);
            x[i] = i < lane ? 0.f : betas[warp][i] * ((i == lane ? 1.f : 0.f) - ik[i] * s);
            mat[i * CHUNK + lane] = x[i];
        }
    }
    for (int e = lane; e < 64; e += 32) {
        const int i = e >> 3, j = e & 7;
        mat[64 + e] = j <= i ? sum[28 + i * (i + 1) / 2 + j] * iq[i] * ik[j] : 0.f;
    }
    for (int d = lane; d < a.vdim; d += 32) {
        float v[CHUNK];
        convolve_chunk(2 * kd + h * a.vdim + d, v);
#pragma unroll
        for (int j = 0; j < CHUNK; j++)
            if (j < count) values[(size_t)(run.x - first + c0 + j) * value_ld(a) + h * a.vdim + d] = v[j];
    }
}

// A number as two tf32 parts (10 bits behind the leading one), the first rounded to nearest; of the second the product drops what is below
// its own 10 bits.
__device__ __forceinline__ void split_tf32(float v, uint32_t& hi, uint32_t& lo) {
    hi = (__float_as_uint(v) + 0x1000u) & 0xffffe000u;
    lo = __float_as_uint(v - __uint_as_float(hi));
}
__device__ __forceinline__ void mma_tf32(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Accumulators as a left operand
__device__ __forceinline__ void split_rows(const float (&c)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
    split_tf32(c[0], hi[0], lo[0]);
    split_tf32(c[2], hi[1], lo[1]);
    split_tf32(c[1], hi[2], lo[2]);
    split_tf32(c[3], hi[3], lo[3]);
}

constexpr int SCAN_COLS = 16, SCAN_WARPS = 4;          // columns of a CTA; warps that share the key channels

// grid = (column slices, heads, runs); SCAN_STAGES: packets under way. A CTA keeps 16 columns of a state, each warp TILES tiles of 8 key channels of them. Lane (g, t):
// columns g and g + 8, channels 2t and 2t + 1 of every tile, tokens 2t and 2t + 1 of a chunk.
template <int TILES, int SCAN_STAGES>
__global__ void __launch_bounds__(SCAN_WARPS * 32)
delta_scan_kernel(const cmlb200_delta a, const float* __restrict__ proj, int ld, const int* __restrict__ row_pos, const int4* __restrict__ runs, int first,
                  float* __restrict__ values, const float* __restrict__ packets) {
    extern __shared__ __align__(16) float stage[];
    constexpr int ALL = TILES * SCAN_WARPS, FLOATS = ALL * 200 + 144, AHEAD = 3;            // AHEAD: chunks whose values are under way
    __shared__ __align__(16) float4 part[2][SCAN_WARPS][2][32];        // the warps' shares of both sums, by turns
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.y, group = a.heads / a.kv_heads, kh = h / group, vld = value_ld(a);
    const int col = blockIdx.x * SCAN_COLS + g, d0 = warp * TILES * 8;
    dep_wait();
    const int4 run = runs[blockIdx.z];
    const int n = run.y, slot = run.z, p0 = row_pos[run.x], chunks = (n + CHUNK - 1) / CHUNK;
    const float* src = packets + ((size_t)first_packet(run, blockIdx.z, first) * a.heads + h) * FLOATS;
    float* vrow = values + (size_t)(run.x - first) * vld + h * a.vdim;
    auto fetch = [&](int c) {
        if (c < chunks) {
            const float* from = src + (size_t)c * a.heads * FLOATS;
            float* to = stage + (c % SCAN_STAGES) * FLOATS;
#pragma unroll 8
            for (int i = tid * 4; i < FLOATS; i += SCAN_WARPS * 32 * 4) cp16(smem_addr(to + i), from + i);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    auto fetch_values = [&](int c, float (&v)[4]) {
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int tok = c * CHUNK + 2 * t + (e & 1), cc = col + (e >> 1) * 8;
            v[e] = tok < n && cc < a.vdim ? vrow[(size_t)tok * vld + cc] : 0.f;
        }
    };
    for (int c = 0; c < SCAN_STAGES - 1; c++) fetch(c);
    float v_next[AHEAD][4];
#pragma unroll
    for (int k = 0; k < AHEAD; k++) fetch_values(k, v_next[k]);
    float S[TILES][4];
    float* state = a.state + ((size_t)slot * a.heads + h) * a.dim * a.vdim_ld;
#pragma unroll
    for (int i = 0; i < TILES; i++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int d = d0 + i * 8 + 2 * t + (e & 1), cc = col + (e >> 1) * 8;
            S[i][e] = p0 > 0 && d < a.dim && cc < a.vdim ? state[(size_t)d * a.vdim_ld + cc] : 0.f;
        }
    if (blockIdx.x == 0) {                             // the latest projections; nobody reads the ring in this launch
        const int keep = min(n, a.taps - 1), kd = a.kv_heads * a.dim, channels = delta_channels(a);
        for (int k = n - keep; k < n; k++) {
            float* ring = a.ring + ((size_t)slot * a.taps + (p0 + k) % a.taps) * channels;
            const float* row = proj + (size_t)(run.x + k) * ld + a.col;
            if (h == kh * group)
                for (int d = tid; d < a.dim; d += blockDim.x) {
                    ring[kh * a.dim + d] = row[kh * a.dim + d];
                    ring[kd + kh * a.dim + d] = row[kd + kh * a.dim + d];
                }
            for (int d = tid; d < a.vdim; d += blockDim.x) ring[2 * kd + h * a.vdim + d] = row[2 * kd + h * a.vdim + d];
        }
    }
    for (int c = 0; c < chunks; c++) {
        asm volatile("cp.async.wait_group %0;" ::"n"(SCAN_STAGES - 2) : "memory");
        __syncthreads();                               // this chunk is there, and the one before it is read
        const float* st = stage + (c % SCAN_STAGES) * FLOATS;
        const float *kq = st + warp * TILES * 128, *kt = st + ALL * 128 + warp * TILES * 64, *gt = st + ALL * 192 + d0, *mat = st + ALL * 200;
        float rk[3][4] = {}, rq[3][4] = {};
#pragma unroll
        for (int i = 0; i < TILES; i++) {
            const float4 x = *reinterpret_cast<const float4*>(kq + i * 128 + g * 16 + t * 4);
            uint32_t hi[4], lo[4], k0, k1, l0, l1, q0, q1, m0, m1;
            split_rows(S[i], hi, lo);
            split_tf32(x.x, k0, l0);
            split_tf32(x.y, k1, l1);
            split_tf32(x.z, q0, m0);
            split_tf32(x.w, q1, m1);
            mma_tf32(rk[0], hi, k0, k1);
            mma_tf32(rq[0], hi, q0, q1);
            mma_tf32(rk[1], hi, l0, l1);
            mma_tf32(rq[1], hi, m0, m1);
            mma_tf32(rk[2], lo, k0, k1);
            mma_tf32(rq[2], lo, q0, q1);
        }
        float v[4];
#pragma unroll
        for (int e = 0; e < 4; e++) {
            v[e] = v_next[0][e];
#pragma unroll
            for (int k = 1; k < AHEAD; k++) v_next[k - 1][e] = v_next[k][e];
            rk[0][e] += rk[1][e] + rk[2][e];
            rq[0][e] += rq[1][e] + rq[2][e];
        }
        part[c & 1][warp][0][lane] = make_float4(rk[0][0], rk[0][1], rk[0][2], rk[0][3]);
        part[c & 1][warp][1][lane] = make_float4(rq[0][0], rq[0][1], rq[0][2], rq[0][3]);
        fetch(c + SCAN_STAGES - 1);                    // into the stage that the barrier above released
        fetch_values(c + AHEAD, v_next[AHEAD - 1]);
        __syncthreads();
        const float2 ik = *reinterpret_cast<const float2*>(mat + 128 + 2 * t), iq = *reinterpret_cast<const float2*>(mat + 136 + 2 * t);
        float4 k = part[c & 1][0][0][lane], q = part[c & 1][0][1][lane];
#pragma unroll
        for (int w = 1; w < SCAN_WARPS; w++) {
            const float4 x = part[c & 1][w][0][lane], y = part[c & 1][w][1][lane];
            k.x += x.x; k.y += x.y; k.z += x.z; k.w += x.w;
            q.x += y.x; q.y += y.y; q.z += y.z; q.w += y.w;
        }
        const float x[4] = {fmaf(-ik.x, k.x, v[0]), fmaf(-ik.y, k.y, v[1]), fmaf(-ik.x, k.z, v[2]), fmaf(-ik.y, k.w, v[3])};
        uint32_t hi[4], lo[4], b0, b1, c0, c1;
        float u[4] = {}, u1[4] = {}, u2[4] = {};
        float2 m = *reinterpret_cast<const float2*>(mat + g * 8 + 2 * t);
        split_rows(x, hi, lo);
        split_tf32(m.x, b0, c0);
        split_tf32(m.y, b1, c1);
        mma_tf32(u, hi, b0, b1);
        mma_tf32(u1, hi, c0, c1);
        mma_tf32(u2, lo, b0, b1);
#pragma unroll
        for (int e = 0; e < 4; e++) u[e] += u1[e] + u2[e];
        if (warp == (c & (SCAN_WARPS - 1))) {          // the output, a chunk each in turn
            float o[4] = {iq.x * q.x, iq.y * q.y, iq.x * q.z, iq.y * q.w}, o1[4] = {}, o2[4] = {};
            m = *reinterpret_cast<const float2*>(mat + 64 + g * 8 + 2 * t);
            split_rows(u, hi, lo);
            split_tf32(m.x, b0, c0);
            split_tf32(m.y, b1, c1);
            mma_tf32(o, hi, b0, b1);
            mma_tf32(o1, hi, c0, c1);
            mma_tf32(o2, lo, b0, b1);
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int tok = c * CHUNK + 2 * t + (e & 1), cc = col + (e >> 1) * 8;
                if (tok < n && cc < a.vdim) vrow[(size_t)tok * vld + cc] = o[e] + (o1[e] + o2[e]);
            }
        }
        u[0] *= ik.x; u[1] *= ik.y; u[2] *= ik.x; u[3] *= ik.y;
        split_rows(u, hi, lo);
        constexpr int AT_ONCE = TILES < 4 ? TILES : 4; // a tile's three products wait for one another
#pragma unroll
        for (int i = 0; i < TILES; i += AT_ONCE) {
            uint32_t k0[AT_ONCE], k1[AT_ONCE], l0[AT_ONCE], l1[AT_ONCE];
#pragma unroll
            for (int j = 0; j < AT_ONCE; j++) {
                const float2 y = *reinterpret_cast<const float2*>(kt + (i + j) * 64 + g * 8 + 2 * t), f = *reinterpret_cast<const float2*>(gt + (i + j) * 8 + 2 * t);
                split_tf32(y.x, k0[j], l0[j]);
                split_tf32(y.y, k1[j], l1[j]);
                S[i + j][0] *= f.x; S[i + j][1] *= f.y; S[i + j][2] *= f.x; S[i + j][3] *= f.y;
            }
#pragma unroll
            for (int j = 0; j < AT_ONCE; j++) mma_tf32(S[i + j], hi, k0[j], k1[j]);
#pragma unroll
            for (int j = 0; j < AT_ONCE; j++) mma_tf32(S[i + j], hi, l0[j], l1[j]);
#pragma unroll
            for (int j = 0; j < AT_ONCE; j++) mma_tf32(S[i + j], lo, k0[j], k1[j]);
        }
    }
    dep_trigger();
#pragma unroll
    for (int i = 0; i < TILES; i++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int d = d0 + i * 8 + 2 * t + (e & 1), cc = col + (e >> 1) * 8;
            if (d < a.dim && cc < a.vdim) state[(size_t)d * a.vdim_ld + cc] = S[i][e];
        }
}

// W: 4 where value rows, gates and outputs allow four columns at a time, else 1
template <typename TO, int W>
__global__ void __launch_bounds__(256)
delta_output_kernel(const cmlb200_delta a, const float* __restrict__ values, const float* __restrict__ gate, int ld_gate, int first, TO* __restrict__ out, int out_ld) {
    constexpr int N = 8 / W;                           // vdim up to 256
    dep_wait();
    dep_trigger();
    const int h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, r = first + blockIdx.x;
    if (h >= a.heads) return;
    const float* o = values + (size_t)blockIdx.x * value_ld(a) + h * a.vdim;
    const float* g = gate + (size_t)r * ld_gate + h * a.vdim;
    TO* dst = out + (size_t)r * out_ld + h * a.vdim;
    float v[N][W], z[N][W], ss = 0.f;
#pragma unroll
    for (int i = 0; i < N; i++) {
        const int d = (lane + 32 * i) * W;
        const bool have = d < a.vdim;
        if constexpr (W == 4) {
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f), x = have ? *reinterpret_cast<const float4*>(o + d) : zero, y = have ? *reinterpret_cast<const float4*>(g + d) : zero;
            v[i][0] = x.x; v[i][1] = x.y; v[i][2] = x.z; v[i][3] = x.w;
            z[i][0] = y.x; z[i][1] = y.y; z[i][2] = y.z; z[i][3] = y.w;
        } else {
            v[i][0] = have ? o[d] : 0.f;
            z[i][0] = have ? g[d] : 0.f;
        }
#pragma unroll
        for (int e = 0; e < W; e++) ss = fmaf(v[i][e], v[i][e], ss);
    }
    const float inv = delta_scale(a) / sqrtf(lane_sum(ss) / (float)a.vdim + a.eps);
#pragma unroll
    for (int i = 0; i < N; i++) {
        const int d = (lane + 32 * i) * W;
        if (d >= a.vdim) continue;
        TO n[W];
#pragma unroll
        for (int e = 0; e < W; e++) n[e] = narrow<TO>(v[i][e] * inv * a.norm[d + e] * sigmoid_fast(z[i][e]));
        if constexpr (W == 4) {
            if constexpr (sizeof(TO) == 2) *reinterpret_cast<uint2*>(dst + d) = *reinterpret_cast<const uint2*>(n);
            else *reinterpret_cast<float4*>(dst + d) = *reinterpret_cast<const float4*>(n);
        } else {
            dst[d] = n[0];
        }
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
    while (splits < 8 && cols > 16 && (rpt > 8 || (long long)rows * a->heads * splits < 2 * cmlb_num_sms())) rpt = shape(splits *= 2, cols, lanes);
    CMLB_REQUIRE(rpt <= 32, "cmlb200_delta_one: states of %d x %d", a->dim, a->vdim);
    const size_t smem = sizeof(float) * ((size_t)3 * ((a->dim + 3) & ~3) + cols + (size_t)8 * lanes * 8 + 8);
    const dim3 grid(splits, a->heads, rows);
#define DO_LAUNCH(TO, RPT, T) CMLB_CUDA(launch_chain(delta_one_kernel<TO, RPT, T>, grid, dim3(ONE_THREADS), smem, splits, as_stream(stream), *a, d_proj, ld, d_decay, \
                                                     ld_decay, d_gate, ld_gate, d_row_pos, d_row_slot, cols, lanes, (TO*)d_out, out_ld))
#define DO_TAPS(TO, RPT) do { if (a->taps == 4) DO_LAUNCH(TO, RPT, 4); else DO_LAUNCH(TO, RPT, 0); } while (0)
#define DO_ROWS(TO) do { if (rpt <= 4) DO_TAPS(TO, 4); else if (rpt <= 8) DO_TAPS(TO, 8); else if (rpt <= 16) DO_TAPS(TO, 16); else DO_TAPS(TO, 32); } while (0)
    if (out_dtype == CMLB200_DT_BF16) DO_ROWS(__nv_bfloat16);
    else DO_ROWS(float);
#undef DO_ROWS
#undef DO_TAPS
#undef DO_LAUNCH
    return CMLB200_OK;
}

extern "C" long cmlb200_delta_work_floats(const cmlb200_delta* a, int rows, int runs) {
    return a ? (long)rows * value_ld(*a) + (long)(rows / CHUNK + runs) * a->heads * packet_floats(scan_tiles(*a)) : 0;
}

extern "C" int cmlb200_delta_rows(const cmlb200_delta* a, const float* d_proj, int ld, const float* d_decay, int ld_decay, const float* d_gate, int ld_gate,
                                  const int* d_row_pos, const int* d_row_slot, int first, int rows, const int* d_runs, int runs, float* d_work, void* d_out,
                                  int out_dtype, int out_ld, void* stream) {
    const int rc = delta_check(a, d_proj, ld, d_decay, ld_decay, d_gate, ld_gate, d_row_pos, d_row_slot, 1, d_out, out_dtype, out_ld, "cmlb200_delta_rows");
    if (rc) return rc;
    CMLB_REQUIRE((long long)rows * ld < (1ll << 31), "cmlb200_delta_rows: %d rows of %d", rows, ld);
    CMLB_REQUIRE(d_runs && runs > 0 && runs <= 65535 && rows > 0 && first >= 0 && d_work && (((uintptr_t)d_runs | (uintptr_t)d_work) & 15) == 0, "cmlb200_delta_rows: bad argument");
    cudaStream_t st = as_stream(stream);
    const int tiles = scan_tiles(*a);
    float* packets = d_work + (size_t)rows * value_ld(*a);
    const dim3 grid(rows / CHUNK + runs, (a->heads + 3) / 4);
#define DP_LAUNCH(T) CMLB_CUDA(launch_chain(delta_prepare_kernel<T>, grid, dim3(128), 0, 1, st, *a, d_proj, ld, d_decay, ld_decay, d_row_pos, (const int4*)d_runs, runs, first, \
                                            d_work, packets))
    if (a->taps == 4) DP_LAUNCH(4);
    else DP_LAUNCH(0);
#undef DP_LAUNCH
    const dim3 grid_scan((a->vdim + SCAN_COLS - 1) / SCAN_COLS, a->heads, runs);
    // few CTAs: each has to cover the latency of its packets alone; many: more of them fit an SM
    const bool deep = (long long)grid_scan.x * grid_scan.y * grid_scan.z <= 2 * cmlb_num_sms();
    static size_t attr[8][kMaxDevices] = {};
#define DS_LAUNCH(N, STAGES, slot)                                                                                                  \
    do {                                                                                                                            \
        auto kern = delta_scan_kernel<N, STAGES>;                                                                                   \
        const size_t smem = (size_t)STAGES * packet_floats(tiles) * sizeof(float);                                                  \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                        \
        CMLB_CUDA(launch_chain(kern, grid_scan, dim3(SCAN_WARPS * 32), smem, 1, st, *a, d_proj, ld, d_row_pos, (const int4*)d_runs, first, d_work, (const float*)packets)); \
    } while (0)
#define DS_DEPTH(N, slot) do { if (deep) DS_LAUNCH(N, (N > 4 ? 4 : 6), slot); else DS_LAUNCH(N, 3, slot + 1); } while (0)
    if (tiles == 4) DS_DEPTH(1, 0);
    else if (tiles == 8) DS_DEPTH(2, 2);
    else if (tiles == 16) DS_DEPTH(4, 4);
    else DS_DEPTH(8, 6);
#undef DS_DEPTH
#undef DS_LAUNCH
    const dim3 grid_out(rows, (a->heads + 7) / 8);
    const bool vec = a->vdim % 4 == 0 && ld_gate % 4 == 0 && out_ld % 4 == 0 && (((uintptr_t)d_gate | (uintptr_t)d_out) & 15) == 0;
#define DU_LAUNCH(TO, W) CMLB_CUDA(launch_chain(delta_output_kernel<TO, W>, grid_out, dim3(256), 0, 1, st, *a, (const float*)d_work, d_gate, ld_gate, first, (TO*)d_out, out_ld))
    if (out_dtype == CMLB200_DT_BF16) { if (vec) DU_LAUNCH(__nv_bfloat16, 4); else DU_LAUNCH(__nv_bfloat16, 1); }
    else { if (vec) DU_LAUNCH(float, 4); else DU_LAUNCH(float, 1); }
#undef DU_LAUNCH
    return CMLB200_OK;
}
