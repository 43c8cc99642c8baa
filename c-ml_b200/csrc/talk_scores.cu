// Scores of layers whose heads see one another's: score_h = sum_g talk[h][g] c(q_g . k_g scale), c(s) = cap tanh(s / cap). All
// heads of a (query, key) pair have to be known before any of them may enter a softmax, so the scores get a pass
// of their own, fp32 in global memory, which the attention kernels (attention_rows.cu, cmlb200_attn's `scores`) then read in
// place of computing q . k. Queries are those of cmlb200_rotate_append, keys are in the cache.
//
//   talk_tiles_kernel   prompt portions: a CTA computes QN queries x KN keys of every head on mma.sync m16n8k16 straight
//                       from global memory into shared memory, then mixes: a thread keeps 8 heads x 4 keys in registers
//                       and walks over the heads that speak. The mixing is fp32 throughout
//   talk_rows_kernel    decoded tokens (fp16 cache) and any rows of the 32-bit form: a lane per key, 32 keys to a CTA
//
// Over an fp16 cache the scores leave in units of log2, as those kernels want them. Blocks of keys that no row of a tile
// sees are skipped; which keys a row sees within a block is the reader's business.
#include "lm_util.cuh"

namespace {

__device__ __forceinline__ int talk_first_key(const cmlb200_attn& a, int p) { return (a.window > 0 && a.window <= p) ? p - a.window + 1 : 0; }
// tanh from the hardware exponential: an error of a few units of 2^-24, which the cap multiplies
__device__ __forceinline__ float cap_fast(float s, float cap, float inv) { return cap - __fdividef(2.0f * cap, 1.0f + __expf(2.0f * inv * s)); }

constexpr int TT_THREADS = 256, TT_WARPS = TT_THREADS / 32;

// Column c of row r lies at r * KN + (c ^ talk_swizzle(r)): neighbouring rows start at other banks.
template <int KN> __device__ __forceinline__ int talk_swizzle(int r) { return KN == 32 ? (r & 3) << 3 : ((r >> 1) & 1) << 3; }

// grid = (key blocks, 64 / QN, tiles). scores: [tile][heads][64][ld], keys from that of the tile's first row rounded down to 16.
template <int QN, int KN>
__global__ void __launch_bounds__(TT_THREADS)
talk_tiles_kernel(const cmlb200_attn a, const __half* __restrict__ q, const int4* __restrict__ tiles, float* __restrict__ scores, int ld) {
    extern __shared__ __align__(16) float sc[];        // [heads][QN * KN], then talk transposed [heads][heads rounded up to 8]
    constexpr int QM = QN / 16, KM = KN / 8, PAIRS = QN * KN;
    dep_wait();
    dep_trigger();
    const int4 tl = tiles[blockIdx.z];
    const int n = tl.y, q0 = blockIdx.y * QN, p_last = tl.w + n - 1;
    if (q0 >= n) return;
    const int k_lo = talk_first_key(a, tl.w) & ~15, kt = k_lo + blockIdx.x * KN, q_last = min(q0 + QN, n) - 1;
    if (kt > tl.w + q_last || kt + KN <= talk_first_key(a, tl.w + q0)) return;
    const int H = a.heads, h8 = (H + 7) & ~7, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
    const int shift = __ffs(a.block_size) - 1, group = H / a.kv_heads;
    const int* table = a.block_table + (size_t)tl.z * a.table_ld;
    float* mix = sc + (size_t)H * PAIRS;
    if (a.talk)
        for (int i = threadIdx.x; i < H * h8; i += TT_THREADS) { const int from = i / h8, to = i - from * h8; mix[i] = to < H ? a.talk[to * H + from] : 0.f; }
    // this lane's rows of both operands; those past the portion's end repeat the last, and nobody reads their scores
    const __half* qr[2 * QM];
    const __half* kr[KM];
#pragma unroll
    for (int i = 0; i < 2 * QM; i++) qr[i] = q + (size_t)(tl.x + min(q0 + i * 8 + g, n - 1)) * H * a.dim_ld + 8 * t;
#pragma unroll
    for (int j = 0; j < KM; j++) {
        const int key = min(kt + j * 8 + g, p_last);
        kr[j] = static_cast<const __half*>(a.k_pool) + (((size_t)table[key >> shift] << shift) + (key & (a.block_size - 1))) * a.kv_heads * a.dim_ld + 8 * t;
    }
    const float inv = a.cap > 0.f ? 1.0f / a.cap : 0.f;
    for (int h = warp; h < H; h += TT_WARPS) {
        const int qo = h * a.dim_ld, ko = h / group * a.dim_ld;
        float s[QM][KM][4];
#pragma unroll
        for (int i = 0; i < QM; i++)
#pragma unroll
            for (int j = 0; j < KM; j++) { s[i][j][0] = 0.f; s[i][j][1] = 0.f; s[i][j][2] = 0.f; s[i][j][3] = 0.f; }
        // any order of the columns will do when both operands use the same: 16 bytes per row and 32 columns feed two products
#pragma unroll 2
        for (int c = 0; c < a.dim_ld; c += 32) {
            const bool have = c + 8 * t < a.dim_ld;
            uint4 qa[2 * QM], kb[KM];
#pragma unroll
            for (int i = 0; i < 2 * QM; i++) qa[i] = have ? *reinterpret_cast<const uint4*>(qr[i] + qo + c) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
            for (int j = 0; j < KM; j++) kb[j] = have ? *reinterpret_cast<const uint4*>(kr[j] + ko + c) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
            for (int i = 0; i < QM; i++) {
                const uint32_t lo[4] = {qa[2 * i].x, qa[2 * i + 1].x, qa[2 * i].y, qa[2 * i + 1].y}, hi[4] = {qa[2 * i].z, qa[2 * i + 1].z, qa[2 * i].w, qa[2 * i + 1].w};
#pragma unroll
                for (int j = 0; j < KM; j++) {
                    mma_f16(s[i][j], lo, kb[j].x, kb[j].y);
                    mma_f16(s[i][j], hi, kb[j].z, kb[j].w);
                }
            }
        }
        float* d = sc + (size_t)h * PAIRS;
#pragma unroll
        for (int i = 0; i < QM; i++)
#pragma unroll
            for (int j = 0; j < KM; j++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int r = i * 16 + e * 8 + g;
                    float2 v = make_float2(s[i][j][2 * e] * a.scale, s[i][j][2 * e + 1] * a.scale);
                    if (a.cap > 0.f) v = make_float2(cap_fast(v.x, a.cap, inv), cap_fast(v.y, a.cap, inv));
                    *reinterpret_cast<float2*>(d + r * KN + ((j * 8 + 2 * t) ^ talk_swizzle<KN>(r))) = v;
                }
    }
    __syncthreads();
    constexpr int QUADS = PAIRS / 4;
    for (int u = threadIdx.x; u < QUADS * (h8 / 8); u += TT_THREADS) {
        const int hb = u / QUADS * 8, quad = u % QUADS, r = quad / (KN / 4), c = quad % (KN / 4) * 4, at = r * KN + (c ^ talk_swizzle<KN>(r));
        if (q0 + r >= n) continue;
        float4 y[8];
        if (a.talk) {
#pragma unroll
            for (int i = 0; i < 8; i++) y[i] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
            for (int f = 0; f < H; f++) {
                const float4 v = *reinterpret_cast<const float4*>(sc + (size_t)f * PAIRS + at);
                const float4 w0 = *reinterpret_cast<const float4*>(mix + f * h8 + hb), w1 = *reinterpret_cast<const float4*>(mix + f * h8 + hb + 4);
                const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
                for (int i = 0; i < 8; i++) {
                    y[i].x = fmaf(w[i], v.x, y[i].x); y[i].y = fmaf(w[i], v.y, y[i].y); y[i].z = fmaf(w[i], v.z, y[i].z); y[i].w = fmaf(w[i], v.w, y[i].w);
                }
            }
        } else {
#pragma unroll
            for (int i = 0; i < 8; i++) y[i] = *reinterpret_cast<const float4*>(sc + (size_t)min(hb + i, H - 1) * PAIRS + at);
        }
        float* out = scores + (((size_t)blockIdx.z * H + hb) * 64 + q0 + r) * ld + (kt - k_lo) + c;
#pragma unroll
        for (int i = 0; i < 8; i++)
            if (hb + i < H) *reinterpret_cast<float4*>(out + (size_t)i * 64 * ld) = make_float4(y[i].x * kLog2e, y[i].y * kLog2e, y[i].z * kLog2e, y[i].w * kLog2e);
    }
}

template <typename KV> struct Chunk8;                  // eight elements of a cached key as fp32
template <> struct Chunk8<__half> {
    uint4 w;
    __device__ __forceinline__ void load(const __half* p) { w = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ float dot(const float* q, float s) const {
        const uint32_t u[4] = {w.x, w.y, w.z, w.w};
        const float4 x = *reinterpret_cast<const float4*>(q), y = *reinterpret_cast<const float4*>(q + 4);
        const float b[8] = {x.x, x.y, x.z, x.w, y.x, y.y, y.z, y.w};
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const float2 k = __half22float2(*reinterpret_cast<const __half2*>(&u[i]));
            s = fmaf(b[2 * i], k.x, fmaf(b[2 * i + 1], k.y, s));
        }
        return s;
    }
};
template <> struct Chunk8<float> {
    float4 u, v;
    __device__ __forceinline__ void load(const float* p) { u = *reinterpret_cast<const float4*>(p); v = *reinterpret_cast<const float4*>(p + 4); }
    __device__ __forceinline__ float dot(const float* q, float s) const {
        const float4 x = *reinterpret_cast<const float4*>(q), y = *reinterpret_cast<const float4*>(q + 4);
        s = fmaf(x.x, u.x, fmaf(x.y, u.y, fmaf(x.z, u.z, fmaf(x.w, u.w, s))));
        return fmaf(y.x, v.x, fmaf(y.y, v.y, fmaf(y.z, v.z, fmaf(y.w, v.w, s))));
    }
};

constexpr int TR_KEYS = 32, TR_LD = TR_KEYS + 1;

// grid = (key blocks, rows). scores: [row][heads][ld], keys from the first one the row sees.
template <typename KV>
__global__ void __launch_bounds__(512)
talk_rows_kernel(const cmlb200_attn a, const KV* __restrict__ q, const int* __restrict__ row_pos, const int* __restrict__ row_slot, float* __restrict__ scores, int ld) {
    extern __shared__ __align__(16) float sm[];
    const int H = a.heads, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    float *q_s = sm, *sc = q_s + H * a.dim_ld;         // [heads][dim_ld], [heads][TR_LD]
    dep_wait();
    dep_trigger();
    const int r = blockIdx.y, p = row_pos[r], k_lo = talk_first_key(a, p), seen = p + 1 - k_lo, k0 = blockIdx.x * TR_KEYS;
    if (k0 >= seen) return;
    const int shift = __ffs(a.block_size) - 1, group = H / a.kv_heads;
    const int key = k_lo + min(k0 + lane, seen - 1);
    const KV* kr = static_cast<const KV*>(a.k_pool) +
                   (((size_t)a.block_table[(size_t)row_slot[r] * a.table_ld + (key >> shift)] << shift) + (key & (a.block_size - 1))) * a.kv_heads * a.dim_ld;
    for (int i = threadIdx.x; i < H * a.dim_ld; i += blockDim.x) q_s[i] = widen(q[(size_t)r * H * a.dim_ld + i]) * a.scale;
    __syncthreads();
    for (int kh = warp; kh < a.kv_heads; kh += warps) {
        const KV* k = kr + (size_t)kh * a.dim_ld;
        for (int j0 = 0; j0 < group; j0 += 4) {
            const float* qh = q_s + (kh * group + j0) * a.dim_ld;
            float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
            for (int c = 0; c < a.dim_ld; c += 8) {
                Chunk8<KV> w;
                w.load(k + c);
#pragma unroll
                for (int j = 0; j < 4; j++)
                    if (j0 + j < group) s[j] = w.dot(qh + j * a.dim_ld + c, s[j]);
            }
#pragma unroll
            for (int j = 0; j < 4; j++)
                if (j0 + j < group) sc[(kh * group + j0 + j) * TR_LD + lane] = a.cap > 0.f ? soft_cap(s[j], a.cap) : s[j];
        }
    }
    __syncthreads();
    for (int h = warp; h < H; h += warps) {
        float y = 0.f;
        if (a.talk) {
            const float* w = a.talk + (size_t)h * H;
#pragma unroll 8
            for (int f = 0; f < H; f++) y = fmaf(w[f], sc[f * TR_LD + lane], y);
        } else {
            y = sc[h * TR_LD + lane];
        }
        if (k0 + lane < seen) scores[((size_t)r * H + h) * ld + k0 + lane] = sizeof(KV) == 2 ? y * kLog2e : y;
    }
}

int check_talk(const cmlb200_attn* a, const void* q, const float* scores, int ld, const char* who) {
    const int rc = cmlb200_attn_check_(a, who);
    if (rc) return rc;
    CMLB_REQUIRE(q && scores && ld > 0 && ld % 4 == 0 && (((uintptr_t)q | (uintptr_t)scores) & 15) == 0, "%s: queries, scores or their stride %d", who, ld);
    CMLB_REQUIRE(!a->slopes && a->chunk == 0 && a->keep == 0, "%s: windows alone", who);
    return CMLB200_OK;
}

size_t tiles_smem(int heads, int pairs) { return 4 * ((size_t)heads * pairs + (size_t)heads * ((heads + 7) & ~7)); }

}  // namespace

extern "C" int cmlb200_talk_scores_heads(void) {
    int h = 1;
    while (tiles_smem(h + 1, 16 * 16) <= 200 * 1024) h++;
    return h;
}

extern "C" int cmlb200_talk_scores_tiles(const cmlb200_attn* a, const uint16_t* d_q_f16, const int* d_tiles, int tiles, int max_keys, float* d_scores, int ld, void* stream) {
    static const char* who = "cmlb200_talk_scores_tiles";
    CMLB_REQUIRE(a && d_tiles && tiles > 0 && tiles <= 65535 && max_keys > 0 && ((uintptr_t)d_tiles & 15) == 0, "%s: bad argument", who);
    const int rc = check_talk(a, d_q_f16, d_scores, ld, who);
    if (rc) return rc;
    CMLB_REQUIRE(a->cache_dtype == CMLB200_DT_F16, "%s: fp16 cache", who);
    // a tile's keys: those in front of its first row (rounded down to 16) and its own
    const int reach = a->window > 0 && a->window - 1 + 64 + 15 < max_keys ? a->window - 1 + 64 + 15 : max_keys;
    CMLB_REQUIRE(ld % 64 == 0 && ld >= reach, "%s: stride %d for %d keys", who, ld, reach);
    static size_t attr[3][kMaxDevices] = {};
#define TT_LAUNCH(QN, KN, slot)                                                                                                        \
    do {                                                                                                                               \
        auto kern = talk_tiles_kernel<QN, KN>;                                                                                         \
        const size_t smem = tiles_smem(a->heads, QN * KN);                                                                             \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                           \
        CMLB_CUDA(launch_chain(kern, dim3((reach + KN - 1) / KN, 64 / QN, tiles), dim3(TT_THREADS), smem, 1, as_stream(stream), *a, (const __half*)d_q_f16, \
                               (const int4*)d_tiles, d_scores, ld));                                                                   \
    } while (0)
    if (tiles_smem(a->heads, 32 * 32) <= 200 * 1024) TT_LAUNCH(32, 32, 0);
    else if (tiles_smem(a->heads, 32 * 16) <= 200 * 1024) TT_LAUNCH(32, 16, 1);
    else {
        CMLB_REQUIRE(tiles_smem(a->heads, 16 * 16) <= 200 * 1024, "%s: the scores of %d heads do not fit shared memory", who, a->heads);
        TT_LAUNCH(16, 16, 2);
    }
#undef TT_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_talk_scores_rows(const cmlb200_attn* a, const void* d_q, const int* d_row_pos, const int* d_row_slot, int rows, int max_keys, float* d_scores, int ld,
                                        void* stream) {
    static const char* who = "cmlb200_talk_scores_rows";
    CMLB_REQUIRE(a && d_row_pos && d_row_slot && rows > 0 && rows <= 65535 && max_keys > 0, "%s: bad argument", who);
    const int rc = check_talk(a, d_q, d_scores, ld, who);
    if (rc) return rc;
    const int reach = a->window > 0 && a->window < max_keys ? a->window : max_keys;
    CMLB_REQUIRE(ld >= reach, "%s: stride %d for %d keys", who, ld, reach);
    const size_t smem = 4 * ((size_t)a->heads * a->dim_ld + (size_t)a->heads * TR_LD);
    CMLB_REQUIRE(smem <= 200 * 1024, "%s: queries of %d heads of %d do not fit shared memory", who, a->heads, a->dim);
    const int threads = a->kv_heads <= 4 ? 128 : (a->kv_heads <= 8 ? 256 : 512);
    const dim3 grid((reach + TR_KEYS - 1) / TR_KEYS, rows);
    static size_t attr[2][kMaxDevices] = {};
#define TR_LAUNCH(KV, slot)                                                                                                            \
    do {                                                                                                                               \
        auto kern = talk_rows_kernel<KV>;                                                                                              \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                           \
        CMLB_CUDA(launch_chain(kern, grid, dim3(threads), smem, 1, as_stream(stream), *a, (const KV*)d_q, d_row_pos, d_row_slot, d_scores, ld)); \
    } while (0)
    if (a->cache_dtype == CMLB200_DT_F32) TR_LAUNCH(float, 0);
    else TR_LAUNCH(__half, 1);
#undef TR_LAUNCH
    return CMLB200_OK;
}
