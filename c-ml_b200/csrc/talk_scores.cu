// Scores of layers whose heads see one another's: score_h = sum_g talk[h][g] c(q_g . k_g scale), c(s) = cap tanh(s / cap). All
// heads of a (query, key) pair have to be known before any of them may enter a softmax, so the scores get a pass
// of their own, fp32 in global memory, which the attention kernels (attention_rows.cu, cmlb200_attn's `scores`) then read in
// place of computing q . k. Queries are those of cmlb200_rotate_append, keys are in the cache.
//
//   talk_tiles_kernel   prompt portions: a CTA computes QN queries x KN keys of every head on mma.sync m16n8k16 straight
//                       from global memory into shared memory, then mixes: a thread keeps 8 heads x 4 keys in registers
//                       and walks over the heads that speak. The mixing is fp32 throughout
//   talk_rows_kernel    decoded tokens, 8 or 32 keys to a CTA. Over an fp16 cache the query heads of a key head are the rows of the
//                       products; the 32-bit form, which serves any rows, multiplies in fp32
//
// Over an fp16 cache the scores leave in units of log2, as those kernels want them. Blocks of keys that no row of a tile
// sees are skipped; which keys a row sees within a block is the reader's business.
#include "lm_util.cuh"

namespace {

__device__ __forceinline__ int talk_first_key(const cmlb200_attn& a, int p) { return (a.window > 0 && a.window <= p) ? p - a.window + 1 : 0; }
// tanh from the hardware exponential: an error of a few units of 2^-24, which the cap multiplies
__device__ __forceinline__ float cap_fast(float s, float cap, float inv) { return cap - __fdividef(2.0f * cap, 1.0f + __expf(2.0f * inv * s)); }

constexpr int TT_THREADS = 512;
constexpr size_t TT_SMEM = 226 * 1024;

// Column c of row r lies at r * KN + (c ^ talk_swizzle(r)): neighbouring rows start at other banks.
template <int KN> __device__ __forceinline__ int talk_swizzle(int r) { return KN == 32 ? (r & 3) << 3 : ((r >> 1) & 1) << 3; }

// two fp32 products and sums at once
__device__ __forceinline__ void fma_pair(uint64_t& y, uint64_t w, uint64_t v) { asm("fma.rn.f32x2 %0, %1, %2, %0;" : "+l"(y) : "l"(w), "l"(v)); }
__device__ __forceinline__ float2 halves_of(uint64_t y) {
    float2 f;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(y));
    return f;
}

// grid = (key blocks, 64 / QN, tiles). scores: [tile][heads][64][ld], keys from that of the tile's first row rounded down to 16.
// WHOLE: dim_ld is a multiple of 32.
template <int QN, int KN, bool WHOLE>
__global__ void __launch_bounds__(TT_THREADS, 1)
talk_tiles_kernel(const cmlb200_attn a, const __half* __restrict__ q, const int4* __restrict__ tiles, float* __restrict__ scores, int ld) {
    extern __shared__ __align__(16) float sc[];        // [heads][QN * KN], then talk transposed and twice over [heads][heads rounded up to 8][2]
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
    float2* mix = reinterpret_cast<float2*>(sc + (size_t)H * PAIRS);
    if (a.talk)
        for (int i = threadIdx.x; i < H * h8; i += TT_THREADS) {
            const int from = i / h8, to = i - from * h8;
            const float w = to < H ? a.talk[to * H + from] : 0.f;
            mix[i] = make_float2(w, w);
        }
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
    for (int h = warp; h < H; h += TT_THREADS / 32) {
        const int qo = h * a.dim_ld, ko = h / group * a.dim_ld;
        float s[QM][KM][4];
#pragma unroll
        for (int i = 0; i < QM; i++)
#pragma unroll
            for (int j = 0; j < KM; j++) { s[i][j][0] = 0.f; s[i][j][1] = 0.f; s[i][j][2] = 0.f; s[i][j][3] = 0.f; }
        // any order of the columns will do when both operands use the same: 16 bytes per row and 32 columns feed two products
#pragma unroll 2
        for (int c = 0; c < a.dim_ld; c += 32) {
            const bool have = WHOLE || c + 8 * t < a.dim_ld;
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
        float* out = scores + (((size_t)blockIdx.z * H + hb) * 64 + q0 + r) * ld + (kt - k_lo) + c;
        if (a.talk) {
            uint64_t y[8][2];
#pragma unroll
            for (int i = 0; i < 8; i++) { y[i][0] = 0u; y[i][1] = 0u; }
#pragma unroll 4
            for (int f = 0; f < H; f++) {
                const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(sc + (size_t)f * PAIRS + at);
                const ulonglong2* w = reinterpret_cast<const ulonglong2*>(mix + f * h8 + hb);
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const ulonglong2 x = w[i];
                    fma_pair(y[2 * i][0], x.x, v.x);
                    fma_pair(y[2 * i][1], x.x, v.y);
                    fma_pair(y[2 * i + 1][0], x.y, v.x);
                    fma_pair(y[2 * i + 1][1], x.y, v.y);
                }
            }
#pragma unroll
            for (int i = 0; i < 8; i++) {
                const float2 lo = halves_of(y[i][0]), hi = halves_of(y[i][1]);
                if (hb + i < H) *reinterpret_cast<float4*>(out + (size_t)i * 64 * ld) = make_float4(lo.x * kLog2e, lo.y * kLog2e, hi.x * kLog2e, hi.y * kLog2e);
            }
        } else {
            for (int i = 0; i < 8 && hb + i < H; i++) {
                const float4 y = *reinterpret_cast<const float4*>(sc + (size_t)(hb + i) * PAIRS + at);
                *reinterpret_cast<float4*>(out + (size_t)i * 64 * ld) = make_float4(y.x * kLog2e, y.y * kLog2e, y.z * kLog2e, y.w * kLog2e);
            }
        }
    }
}

constexpr int TR_HEADS = 8;                            // query heads of a key head whose sums a lane keeps at a time, in the 32-bit form

__device__ __forceinline__ float cap_exact(const cmlb200_attn& a, float s) { return a.cap > 0.f ? soft_cap(s, a.cap) : s; }

// Scores of KN keys against the heads of a key head, a warp's work: fp16, lane (g, t) holds key g of every eight.
template <int KN, typename Row>
__device__ __forceinline__ void talk_products(const cmlb200_attn& a, const __half* __restrict__ q, Row key_row, int kh, int group, float* sc, int ld) {
    constexpr int KM = KN / 8;
    const int lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const __half* kr[KM];
#pragma unroll
    for (int j = 0; j < KM; j++) kr[j] = key_row(j * 8 + g) + (size_t)kh * a.dim_ld + 8 * t;
    for (int h0 = 0; h0 < group; h0 += 16) {
        const __half* q0 = q + (size_t)(kh * group + h0 + g) * a.dim_ld + 8 * t;
        const bool lo_row = h0 + g < group, hi_row = h0 + g + 8 < group;
        float s[KM][4];
#pragma unroll
        for (int j = 0; j < KM; j++) { s[j][0] = 0.f; s[j][1] = 0.f; s[j][2] = 0.f; s[j][3] = 0.f; }
        const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
#pragma unroll (KN == 8 ? 4 : 1)
        for (int c = 0; c < a.dim_ld; c += 32) {
            const bool have = c + 8 * t < a.dim_ld;
            const uint4 x = have && lo_row ? *reinterpret_cast<const uint4*>(q0 + c) : zero, y = have && hi_row ? *reinterpret_cast<const uint4*>(q0 + (size_t)8 * a.dim_ld + c) : zero;
            const uint32_t lo[4] = {x.x, y.x, x.y, y.y}, hi[4] = {x.z, y.z, x.w, y.w};
            uint4 k[KM];
#pragma unroll
            for (int j = 0; j < KM; j++) k[j] = have ? *reinterpret_cast<const uint4*>(kr[j] + c) : zero;
#pragma unroll
            for (int j = 0; j < KM; j++) {
                mma_f16(s[j], lo, k[j].x, k[j].y);
                mma_f16(s[j], hi, k[j].z, k[j].w);
            }
        }
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int h = h0 + g + 8 * e;
            if (h >= group) continue;
            float* d = sc + (kh * group + h) * ld + 2 * t;
#pragma unroll
            for (int j = 0; j < KM; j++) {
                d[j * 8] = cap_exact(a, s[j][2 * e] * a.scale);
                d[j * 8 + 1] = cap_exact(a, s[j][2 * e + 1] * a.scale);
            }
        }
    }
}

// The same in fp32, eight keys and four lanes to a key at a time; q_s: queries times the scale.
template <int KN, typename Row>
__device__ __forceinline__ void talk_products(const cmlb200_attn& a, const float* q_s, Row key_row, int kh, int group, float* sc, int ld) {
    const int lane = threadIdx.x & 31, part = lane & 3;
    for (int k = lane >> 2; k < KN; k += 8) {
        const float* kr = key_row(k) + (size_t)kh * a.dim_ld;
        for (int j0 = 0; j0 < group; j0 += TR_HEADS) {
            const int nj = min(TR_HEADS, group - j0);
            const float* qh = q_s + (kh * group + j0) * a.dim_ld;
            float s[TR_HEADS];
#pragma unroll
            for (int j = 0; j < TR_HEADS; j++) s[j] = 0.f;
            for (int c = part * 8; c < a.dim_ld; c += 32) {
                const float4 u = *reinterpret_cast<const float4*>(kr + c), v = *reinterpret_cast<const float4*>(kr + c + 4);
#pragma unroll
                for (int j = 0; j < TR_HEADS; j++) {
                    if (j >= nj) break;
                    const float4 x = *reinterpret_cast<const float4*>(qh + j * a.dim_ld + c), y = *reinterpret_cast<const float4*>(qh + j * a.dim_ld + c + 4);
                    s[j] = fmaf(x.x, u.x, fmaf(x.y, u.y, fmaf(x.z, u.z, fmaf(x.w, u.w, s[j]))));
                    s[j] = fmaf(y.x, v.x, fmaf(y.y, v.y, fmaf(y.z, v.z, fmaf(y.w, v.w, s[j]))));
                }
            }
#pragma unroll
            for (int j = 0; j < TR_HEADS; j++) {
                if (j >= nj) break;
                float v = s[j];
                v += __shfl_xor_sync(0xffffffffu, v, 1);
                v += __shfl_xor_sync(0xffffffffu, v, 2);
                if (part == 0) sc[(kh * group + j0 + j) * ld + k] = cap_exact(a, v);
            }
        }
    }
}

__host__ __device__ inline size_t rows_smem(int heads, int dim_ld, int kn, bool f32) { return 4 * ((size_t)(f32 ? heads * dim_ld : 0) + (size_t)heads * (kn + 4) + (size_t)heads * (heads + 1)); }

// grid = (key blocks of KN, rows). scores: [row][heads][ld], keys from the first one the row sees.
template <typename KV, int KN>
__global__ void __launch_bounds__(512, 2)
talk_rows_kernel(const cmlb200_attn a, const KV* __restrict__ q, const int* __restrict__ row_pos, const int* __restrict__ row_slot, float* __restrict__ scores, int ld) {
    extern __shared__ __align__(16) float sm[];
    constexpr int LD = KN + 4;
    constexpr bool F32 = sizeof(KV) == 4;
    const int H = a.heads, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    float *sc = sm, *q_s = sc + H * LD, *mix = q_s + (F32 ? H * a.dim_ld : 0);       // [heads][LD], [heads][dim_ld], talk as [heads][heads + 1]
    // neither positions and slots nor blocks come from the launch in front, nor do any keys but the row's own: they are under way
    // to the caches while it ends
    const int r = blockIdx.y, p = row_pos[r], k_lo = talk_first_key(a, p), seen = p + 1 - k_lo, k0 = blockIdx.x * KN;
    if (k0 >= seen) { dep_wait(); return; }
    const int shift = __ffs(a.block_size) - 1, group = H / a.kv_heads, mine = min(KN, seen - k0);
    const int* table = a.block_table + (size_t)row_slot[r] * a.table_ld;
    auto key_row = [&](int k) {
        const int key = k_lo + min(k0 + k, seen - 1);
        return static_cast<const KV*>(a.k_pool) + (((size_t)table[key >> shift] << shift) + (key & (a.block_size - 1))) * a.kv_heads * a.dim_ld;
    };
    const int lines = a.kv_heads * a.dim_ld * (int)sizeof(KV) / 128;
    for (int i = threadIdx.x; i < mine * lines; i += blockDim.x) {
        const char* line = reinterpret_cast<const char*>(key_row(i / lines)) + i % lines * 128;
        asm volatile("prefetch.global.L2 [%0];" ::"l"(line));
    }
    if (a.talk)
        for (int i = threadIdx.x; i < H * H; i += blockDim.x) mix[i / H * (H + 1) + i % H] = a.talk[i];
    dep_wait();
    dep_trigger();
    q += (size_t)r * H * a.dim_ld;
    if constexpr (F32) {
        for (int i = threadIdx.x; i < H * a.dim_ld; i += blockDim.x) q_s[i] = q[i] * a.scale;
        __syncthreads();
    }
    for (int kh = warp; kh < a.kv_heads; kh += warps) {
        if constexpr (F32) talk_products<KN>(a, q_s, key_row, kh, group, sc, LD);
        else talk_products<KN>(a, q, key_row, kh, group, sc, LD);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < H * (KN / 4); i += blockDim.x) {
        const int h = i / (KN / 4), k = i % (KN / 4) * 4;
        float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
        if (a.talk) {
            const float* w = mix + h * (H + 1);
#pragma unroll 8
            for (int f = 0; f < H; f++) {
                const float4 v = *reinterpret_cast<const float4*>(sc + f * LD + k);
                y.x = fmaf(w[f], v.x, y.x); y.y = fmaf(w[f], v.y, y.y); y.z = fmaf(w[f], v.z, y.z); y.w = fmaf(w[f], v.w, y.w);
            }
        } else {
            y = *reinterpret_cast<const float4*>(sc + h * LD + k);
        }
        float* d = scores + ((size_t)r * H + h) * ld + k0 + k;
        const float m = F32 ? 1.f : kLog2e, v[4] = {y.x * m, y.y * m, y.z * m, y.w * m};
        if (k + 4 <= mine) *reinterpret_cast<float4*>(d) = make_float4(v[0], v[1], v[2], v[3]);
        else
            for (int e = 0; e < mine - k; e++) d[e] = v[e];
    }
}

int check_talk(const cmlb200_attn* a, const void* q, const float* scores, int ld, const char* who) {
    const int rc = cmlb200_attn_check_(a, who);
    if (rc) return rc;
    CMLB_REQUIRE(q && scores && ld > 0 && ld % 4 == 0 && (((uintptr_t)q | (uintptr_t)scores) & 15) == 0, "%s: queries, scores or their stride %d", who, ld);
    CMLB_REQUIRE(!a->slopes && a->chunk == 0 && a->keep == 0, "%s: windows alone", who);
    return CMLB200_OK;
}

size_t tiles_smem(int heads, int pairs) { return 4 * ((size_t)heads * pairs + 2 * (size_t)heads * ((heads + 7) & ~7)); }

}  // namespace

extern "C" int cmlb200_talk_scores_heads(void) {
    int h = 1;
    while (tiles_smem(h + 1, 16 * 16) <= TT_SMEM) h++;
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
    static size_t attr[6][kMaxDevices] = {};
#define TT_LAUNCH(QN, KN, WHOLE, slot)                                                                                                 \
    do {                                                                                                                               \
        auto kern = talk_tiles_kernel<QN, KN, WHOLE>;                                                                                  \
        const size_t smem = tiles_smem(a->heads, QN * KN);                                                                             \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                           \
        CMLB_CUDA(launch_chain(kern, dim3((reach + KN - 1) / KN, 64 / QN, tiles), dim3(TT_THREADS), smem, 1, as_stream(stream), *a, (const __half*)d_q_f16, \
                               (const int4*)d_tiles, d_scores, ld));                                                                   \
    } while (0)
#define TT_DIM(QN, KN, slot) do { if (a->dim_ld % 32 == 0) TT_LAUNCH(QN, KN, true, slot); else TT_LAUNCH(QN, KN, false, slot + 1); } while (0)
    if (tiles_smem(a->heads, 32 * 32) <= TT_SMEM) TT_DIM(32, 32, 0);
    else if (tiles_smem(a->heads, 32 * 16) <= TT_SMEM) TT_DIM(32, 16, 2);
    else {
        CMLB_REQUIRE(tiles_smem(a->heads, 16 * 16) <= TT_SMEM, "%s: the scores of %d heads do not fit shared memory", who, a->heads);
        TT_DIM(16, 16, 4);
    }
#undef TT_DIM
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
    // few rows: blocks of eight keys, so that more SMs take part
    const int kn = (long)rows * ((reach + 31) / 32) < 2 * cmlb_num_sms() ? 8 : 32;
    const size_t smem = rows_smem(a->heads, a->dim_ld, kn, a->cache_dtype == CMLB200_DT_F32);
    CMLB_REQUIRE(smem <= 227 * 1024, "%s: queries of %d heads of %d do not fit shared memory", who, a->heads, a->dim);
    const int threads = a->kv_heads <= 4 ? 128 : (a->kv_heads <= 8 ? 256 : 512);
    const dim3 grid((reach + kn - 1) / kn, rows);
    static size_t attr[4][kMaxDevices] = {};
#define TR_LAUNCH(KV, KN, slot)                                                                                                        \
    do {                                                                                                                               \
        auto kern = talk_rows_kernel<KV, KN>;                                                                                          \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                           \
        CMLB_CUDA(launch_chain(kern, grid, dim3(threads), smem, 1, as_stream(stream), *a, (const KV*)d_q, d_row_pos, d_row_slot, d_scores, ld)); \
    } while (0)
    if (a->cache_dtype == CMLB200_DT_F32) { if (kn == 8) TR_LAUNCH(float, 8, 0); else TR_LAUNCH(float, 32, 1); }
    else { if (kn == 8) TR_LAUNCH(__half, 8, 2); else TR_LAUNCH(__half, 32, 3); }
#undef TR_LAUNCH
    return CMLB200_OK;
}
