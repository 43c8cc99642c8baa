// Attention over latents, the mma.sync form for few rows and for what attention_latent_tc.cu does not take, and the entry
// point of both: every head of a row attends the same keys, one vector [latent | rotated part] per token of a
// paged cache, and the weighted sum of the latents is what a head returns. Queries come transformed
// (cmlb200_latent_query), in units of log2. One kernel serves decoded tokens and short prompt portions:
// the (token, head) pairs of a portion are the rows of the matrix products, 16, 32 or 64 to a CTA.
//
// A key tile of 32 tokens is fetched once through the block table (cp.async, two or three stages) and serves both products
// on mma.sync m16n8k16: S = Q K^T with the warps splitting rows, keys and, for few rows, the key columns; O += P K with
// the warps splitting the latent's columns. Scores pass through shared memory, where a few threads per row keep
// the running maximum and sum in fp32. A cluster of up to 16 CTAs splits the keys and merges through distributed
// shared memory, each CTA finishing a share of the values. A tile is a chain of short dependent phases, so the narrow
// form (16 rows) is sized for two CTAs to an SM.
#include "lm_util.cuh"

namespace {

constexpr int LT_THREADS = 256, LT_WARPS = 8, LT_KEYS = 32, LT_SPLITS = 16, LT_SLD = LT_KEYS + 4, LT_PLD = LT_KEYS + 8;

__host__ __device__ constexpr int latent_stages(int rows) { return rows == 16 ? 2 : 3; }
__host__ __device__ inline size_t latent_smem(int rows, int ld, int ldo) {
    const size_t lk = ld + 8;
    const size_t tiles = 2 * lk * (rows + latent_stages(rows) * LT_KEYS), merge = 4 * (size_t)rows * ldo;
    // operands, or the merged values in their place; scores (64 rows of partial sums), weights, per-row factors
    return (tiles > merge ? tiles : merge) + 4 * 64 * LT_SLD + 2 * (size_t)rows * LT_PLD + 3 * 4 * (size_t)rows;
}

// grid = (splits, ceil(tokens * heads / (16 MT)), items), clusters of `splits` CTAs along x. CU: 16-column groups of the
// latent per warp.
template <int MT, int CU>
__global__ void __launch_bounds__(LT_THREADS, MT == 1 ? 2 : 1)
attention_latent_kernel(const cmlb200_latent a, const __half* __restrict__ q, const int* __restrict__ row_pos, const int* __restrict__ row_slot,
                        const int4* __restrict__ tiles, int first, __nv_bfloat16* __restrict__ out) {
    constexpr int MR = 16 * MT, NS = latent_stages(MR), KS = 4 / MT, TPR = LT_THREADS / MR, KPT = LT_KEYS / TPR;
    extern __shared__ __align__(16) uint8_t sm[];
    const int LK = a.ld + 8, rank16 = (a.rank + 15) & ~15, LDO = rank16 + 4;
    __half* Qs = reinterpret_cast<__half*>(sm);
    __half* Ks = Qs + MR * LK;
    const size_t tile_bytes = 2 * (size_t)LK * (MR + NS * LT_KEYS), merge_bytes = 4 * (size_t)MR * LDO;
    float* Ss = reinterpret_cast<float*>(sm + (tile_bytes > merge_bytes ? tile_bytes : merge_bytes));   // [KS][MR][LT_SLD]
    __half* Ps = reinterpret_cast<__half*>(Ss + 64 * LT_SLD);
    float* corr = reinterpret_cast<float*>(Ps + MR * LT_PLD);           // factor on the sums so far, then 1 / sum
    float* c_m = corr + MR;
    float* c_l = c_m + MR;
    float* Os = reinterpret_cast<float*>(sm);                           // [MR][LDO], over the operands once they are done
    dep_wait();
    dep_trigger();
    int4 tl = tiles ? tiles[blockIdx.z] : make_int4((int)blockIdx.z, 1, row_slot[blockIdx.z], row_pos[blockIdx.z]);
    tl.x -= first;
    const int total = tl.y * a.heads, m0 = blockIdx.y * MR;
    if (m0 >= total) return;                                            // the whole cluster leaves
    const int splits = gridDim.x, rank = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
    const int shift = __ffs(a.block_size) - 1;
    const int* table = a.block_table + (size_t)tl.z * a.table_ld;
    const int window = a.window > 0 ? a.window : 0x7fffffff;
    const int p_first = tl.w + m0 / a.heads, p_last = tl.w + (min(m0 + MR, total) - 1) / a.heads;
    const int k_lo = window > p_first ? 0 : p_first - window + 1;
    const int ntiles = (p_last - k_lo) / LT_KEYS + 1;
    const __half* pool = static_cast<const __half*>(a.pool);
    const int kc = a.ld >> 3;

    // a thread copies a part of one key per tile; where that key lies is looked up a tile ahead
    auto slot_of = [&](int it) {
        const int key = min(k_lo + it * LT_KEYS + (int)(threadIdx.x >> 3), p_last);        // past the end: the last key, masked below
        return (table[key >> shift] << shift) + (key & (a.block_size - 1));
    };
    int next_slot = slot_of(rank);
    auto load = [&](int it, int stage) {
        if (it < ntiles) {
            const __half* src = pool + (size_t)next_slot * a.ld;
            const uint32_t dst = smem_addr(Ks + (stage * LT_KEYS + (threadIdx.x >> 3)) * LK);
#pragma unroll 3
            for (int c = threadIdx.x & 7; c < kc; c += 8) cp16(dst + c * 16, src + c * 8);
            next_slot = slot_of(it + splits);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    {
        const __half* src = q + ((size_t)tl.x * a.heads + m0) * a.ld;
        for (int r = threadIdx.x >> 3; r < MR; r += LT_THREADS / 8)
            for (int c = threadIdx.x & 7; c < kc; c += 8) cp16(smem_addr(Qs + r * LK + c * 8), src + (size_t)min(r, total - 1 - m0) * a.ld + c * 8);
    }
#pragma unroll
    for (int i = 0; i < NS - 1; i++) load(rank + i * splits, i);

    float o[MT][CU][2][4];
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int u = 0; u < CU; u++)
#pragma unroll
            for (int e = 0; e < 4; e++) { o[i][u][0][e] = 0.f; o[i][u][1][e] = 0.f; }
    // softmax: thread -> row and keys
    const int sr = threadIdx.x / TPR, sk = (threadIdx.x % TPR) * KPT;
    const int sp = m0 + sr < total ? tl.w + (m0 + sr) / a.heads : -1;
    float m = -INFINITY, l = 0.f;
    // scores: warp -> row tile, 16 keys, share of the columns
    const int w_m = warp % MT, w_k = (warp / MT) & 1, w_s = warp / (2 * MT);
    const uint32_t q_base = smem_addr(Qs + (w_m * 16 + (lane & 15)) * LK + (lane >> 4) * 8);

    int stage = 0;
    for (int it = rank; it < ntiles; it += splits) {
        asm volatile("cp.async.wait_group %0;" ::"n"(NS - 2) : "memory");
        __syncthreads();                                                // this tile is there; the stage of the one before is free
        load(it + (NS - 1) * splits, stage == 0 ? NS - 1 : stage - 1);
        {
            float s[2][4] = {}, s2[2][4] = {};
            const uint32_t k_base = smem_addr(Ks + (stage * LT_KEYS + w_k * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * LK + ((lane >> 3) & 1) * 8);
            // fragments of a step are requested before the products of the one ahead of it
            uint32_t qa[2][4], kb[2][4];
            auto fetch = [&](int kk, int e) {
                ldsm4(q_base + kk * 2, qa[e]);
                ldsm4(k_base + kk * 2, kb[e]);
            };
            constexpr int STEP = KS * 16;
            if (w_s * 16 < a.ld) fetch(w_s * 16, 0);
#pragma unroll 1
            for (int kk = w_s * 16; kk < a.ld; kk += 2 * STEP) {
                if (kk + STEP < a.ld) fetch(kk + STEP, 1);
                mma_f16(s[0], qa[0], kb[0][0], kb[0][1]);
                mma_f16(s[1], qa[0], kb[0][2], kb[0][3]);
                if (kk + STEP >= a.ld) break;
                if (kk + 2 * STEP < a.ld) fetch(kk + 2 * STEP, 0);
                mma_f16(s2[0], qa[1], kb[1][0], kb[1][1]);
                mma_f16(s2[1], qa[1], kb[1][2], kb[1][3]);
            }
#pragma unroll
            for (int j = 0; j < 2; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) s[j][e] += s2[j][e];
            float* d = Ss + (w_s * MR + w_m * 16 + g) * LT_SLD + w_k * 16 + 2 * t;
#pragma unroll
            for (int j = 0; j < 2; j++) {
                *reinterpret_cast<float2*>(d + j * 8) = make_float2(s[j][0], s[j][1]);
                *reinterpret_cast<float2*>(d + j * 8 + 8 * LT_SLD) = make_float2(s[j][2], s[j][3]);
            }
        }
        __syncthreads();
        {
            const int kt = k_lo + it * LT_KEYS;
            float s[KPT], mx = -INFINITY;
#pragma unroll
            for (int j = 0; j < KPT; j++) {
                float v = Ss[sr * LT_SLD + sk + j];
#pragma unroll
                for (int p = 1; p < KS; p++) v += Ss[(p * MR + sr) * LT_SLD + sk + j];
                const int d = sp - (kt + sk + j);
                s[j] = d >= 0 && d < window ? v : -INFINITY;
                mx = fmaxf(mx, s[j]);
            }
#pragma unroll
            for (int w = 1; w < TPR; w <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
            mx = fmaxf(m, mx);
            const float u = mx == -INFINITY ? 0.f : mx, c = ex2(m - u);
            m = mx;
            l *= c;
#pragma unroll
            for (int j = 0; j < KPT; j++) {
                const float e = ex2(s[j] - u);
                l += e;
                Ps[sr * LT_PLD + sk + j] = __float2half_rn(e);
            }
            if (sk == 0) corr[sr] = c;
        }
        __syncthreads();
        {
            uint32_t pa[MT][LT_KEYS / 16][4];
#pragma unroll
            for (int i = 0; i < MT; i++) {
#pragma unroll
                for (int kk = 0; kk < LT_KEYS / 16; kk++) ldsm4(smem_addr(Ps + (i * 16 + (lane & 15)) * LT_PLD + kk * 16 + (lane >> 4) * 8), pa[i][kk]);
                const float c0 = corr[i * 16 + g], c1 = corr[i * 16 + g + 8];
                if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
                    for (int u = 0; u < CU; u++)
#pragma unroll
                        for (int j = 0; j < 2; j++) { o[i][u][j][0] *= c0; o[i][u][j][1] *= c0; o[i][u][j][2] *= c1; o[i][u][j][3] *= c1; }
                }
            }
            const uint32_t v_base = smem_addr(Ks + (stage * LT_KEYS + (lane & 15)) * LK + (lane >> 4) * 8);
            constexpr int KK = LT_KEYS / 16;
            uint32_t vb[2][4];
            auto fetch = [&](int i) {                                   // product i: columns i / KK, keys i % KK
                const int col = (i / KK * LT_WARPS + warp) * 16;
                if (col < rank16) ldsm4_t(v_base + (i % KK * 16 * LK + col) * 2, vb[i & 1]);
            };
            fetch(0);
#pragma unroll
            for (int i = 0; i < CU * KK; i++) {
                if (i + 1 < CU * KK) fetch(i + 1);
                if ((i / KK * LT_WARPS + warp) * 16 < rank16) {
#pragma unroll
                    for (int r = 0; r < MT; r++) {
                        mma_f16(o[r][i / KK][0], pa[r][i % KK], vb[i & 1][0], vb[i & 1][1]);
                        mma_f16(o[r][i / KK][1], pa[r][i % KK], vb[i & 1][2], vb[i & 1][3]);
                    }
                }
            }
        }
        stage = stage == NS - 1 ? 0 : stage + 1;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int w = 1; w < TPR; w <<= 1) l += __shfl_xor_sync(0xffffffffu, l, w);
    __syncthreads();                                                    // every warp is done with the operands and `corr`
    if (sk == 0) {
        c_m[sr] = m;
        c_l[sr] = l;
        const float all = l > 0.f && a.sinks ? l + exp2f(a.sinks[(m0 + sr) % a.heads] * kLog2e - m) : l;      // a sink carries no value
        corr[sr] = all > 0.f ? 1.0f / all : 0.f;
    }
    const size_t out0 = (size_t)tl.x * a.heads + m0;
    if (splits == 1) {
        __syncthreads();
#pragma unroll
        for (int i = 0; i < MT; i++) {
            const int r = i * 16 + g;
            const float i0 = corr[r], i1 = corr[r + 8];
            __nv_bfloat16* d0 = out + (out0 + r) * a.ld_rank;
            __nv_bfloat16* d1 = d0 + (size_t)8 * a.ld_rank;
#pragma unroll
            for (int u = 0; u < CU; u++)
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    const int col = (u * LT_WARPS + warp) * 16 + j * 8 + 2 * t;
                    if (col >= a.rank) continue;
                    // columns rank .. ld_rank meet zero weights; the pair may reach one of them
                    const bool two = col + 1 < a.rank;
                    if (m0 + r < total) *reinterpret_cast<__nv_bfloat162*>(d0 + col) = __floats2bfloat162_rn(o[i][u][j][0] * i0, two ? o[i][u][j][1] * i0 : 0.f);
                    if (m0 + r + 8 < total) *reinterpret_cast<__nv_bfloat162*>(d1 + col) = __floats2bfloat162_rn(o[i][u][j][2] * i1, two ? o[i][u][j][3] * i1 : 0.f);
                }
        }
        return;
    }
#pragma unroll
    for (int i = 0; i < MT; i++)
#pragma unroll
        for (int u = 0; u < CU; u++) {
            const int col = (u * LT_WARPS + warp) * 16 + 2 * t;
            if ((u * LT_WARPS + warp) * 16 < rank16) {
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    *reinterpret_cast<float2*>(Os + (i * 16 + g) * LDO + col + j * 8) = make_float2(o[i][u][j][0], o[i][u][j][1]);
                    *reinterpret_cast<float2*>(Os + (i * 16 + g + 8) * LDO + col + j * 8) = make_float2(o[i][u][j][2], o[i][u][j][3]);
                }
            }
        }
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    const int live = min(MR, total - m0), quads = rank16 / 4;
    for (int i = rank * LT_THREADS + threadIdx.x; i < live * quads; i += splits * LT_THREADS) {
        const int r = i / quads, d = (i - r * quads) * 4;
        float ms[LT_SPLITS], ls[LT_SPLITS];
        float4 xs[LT_SPLITS];
#pragma unroll
        for (int s = 0; s < LT_SPLITS; s++) {
            ms[s] = -INFINITY; ls[s] = 0.f; xs[s] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (s < splits) {
                uint32_t am, al, ax;
                asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(am) : "r"(smem_addr(c_m + r)), "r"(s));
                asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(al) : "r"(smem_addr(c_l + r)), "r"(s));
                asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(ax) : "r"(smem_addr(Os + r * LDO + d)), "r"(s));
                asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(ms[s]) : "r"(am) : "memory");
                asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(ls[s]) : "r"(al) : "memory");
                asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(xs[s].x), "=f"(xs[s].y), "=f"(xs[s].z), "=f"(xs[s].w) : "r"(ax) : "memory");
            }
        }
        float mx = ms[0], sum = 0.f;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int s = 1; s < LT_SPLITS; s++) mx = fmaxf(mx, ms[s]);
#pragma unroll
        for (int s = 0; s < LT_SPLITS; s++) {
            const float c = ms[s] == -INFINITY ? 0.f : exp2f(ms[s] - mx);
            sum = fmaf(ls[s], c, sum);
            x.x = fmaf(xs[s].x, c, x.x); x.y = fmaf(xs[s].y, c, x.y); x.z = fmaf(xs[s].z, c, x.z); x.w = fmaf(xs[s].w, c, x.w);
        }
        if (a.sinks) sum += exp2f(a.sinks[(m0 + r) % a.heads] * kLog2e - mx);
        // columns rank .. ld_rank meet zero weights
        const float inv = 1.0f / sum;
        const __nv_bfloat162 lo = __floats2bfloat162_rn(x.x * inv, d + 1 < a.rank ? x.y * inv : 0.f);
        const __nv_bfloat162 hi = __floats2bfloat162_rn(d + 2 < a.rank ? x.z * inv : 0.f, d + 3 < a.rank ? x.w * inv : 0.f);
        if (d < a.rank)
            *reinterpret_cast<uint2*>(out + (out0 + r) * a.ld_rank + d) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    }
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");      // nobody leaves while others read its shared memory
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}

}  // namespace

static int g_form = 0;
extern "C" int cmlb200_set_attention_latent_form(int form) {
    CMLB_REQUIRE(form >= 0 && form <= 2, "cmlb200_set_attention_latent_form: form %d", form);
    g_form = form;
    return CMLB200_OK;
}

extern "C" double cmlb200_attention_latent_tc_estimate_(const cmlb200_latent* a, int items, int most, int keys, int* splits);
extern "C" int cmlb200_attention_latent_tc_(const cmlb200_latent* a, const uint16_t* q, long q_rows, const int* row_pos, const int* row_slot, int splits,
                                            const int* tiles, int items, int most, int first, uint16_t* o, cudaStream_t st);

extern "C" int cmlb200_attention_latent(const cmlb200_latent* a, const uint16_t* d_q_f16, int q_rows, const int* d_row_pos, const int* d_row_slot, int rows,
                                        int max_keys, const int* d_tiles, int tiles, uint16_t* d_o_bf16, void* stream) {
    static const char* who = "cmlb200_attention_latent";
    CMLB_REQUIRE(a && d_q_f16 && d_o_bf16 && (d_tiles ? tiles > 0 && rows >= 0 : d_row_pos && d_row_slot && rows > 0 && q_rows >= rows) && q_rows > 0 && max_keys >= 0, "%s: bad argument", who);
    CMLB_REQUIRE(a->heads > 0 && a->rank > 0 && a->ld >= a->rank && a->ld % 16 == 0 && a->ld_rank >= a->rank && a->ld_rank % 64 == 0 && a->rank <= 512,
                 "%s: rank %d (up to 512), strides %d / %d", who, a->rank, a->ld, a->ld_rank);
    CMLB_REQUIRE(a->pool && a->block_table && a->table_ld > 0 && a->cache_dtype == CMLB200_DT_F16, "%s: fp16 cache", who);
    CMLB_REQUIRE(a->block_size >= 16 && (a->block_size & (a->block_size - 1)) == 0, "%s: block size %d must be a power of two >= 16", who, a->block_size);
    CMLB_REQUIRE((((uintptr_t)d_q_f16 | (uintptr_t)a->pool | (uintptr_t)d_tiles) & 15) == 0 && ((uintptr_t)d_o_bf16 & 15) == 0, "%s: alignment", who);
    const int items = d_tiles ? tiles : rows, most = d_tiles ? 64 * a->heads : a->heads, sms = cmlb_num_sms();
    CMLB_REQUIRE(items <= 65535, "%s: %d rows", who, items);
    const int keys = (a->window > 0 && a->window < max_keys + 1) ? a->window : max_keys + 1, rank16 = (a->rank + 15) & ~15;
    auto blocks = [&](int m) { return (long)items * ((most + 16 * m - 1) / (16 * m)); };
    // rows per CTA and parts of the keys, by an estimate of the time in microseconds: wide tiles do more per key, narrow
    // ones and more parts spread few heads over more SMs
    int mt = 0, splits = 1;
    double best = 0.0;
    for (int m = 1; m <= 4; m *= 2) {
        const size_t bytes = latent_smem(16 * m, a->ld, rank16 + 4);
        if (bytes > 227 * 1024 || (m > 1 && most <= 8 * m)) continue;
        const long room = (long)sms * (m == 1 && 2 * bytes + 2048 <= 228 * 1024 ? 2 : 1);
        for (int s = 1; s <= (m == 1 ? LT_SPLITS : LT_SPLITS / 2) && (s == 1 || (s - 1) * LT_KEYS < keys); s *= 2) {
            const long ctas = blocks(m) * s, fit = s == LT_SPLITS ? sms : room, waves = (ctas + fit - 1) / fit, tiles_each = ((keys + LT_KEYS - 1) / LT_KEYS + s - 1) / s;
            const double tile = m == 1 ? (ctas > sms ? 2.65 : 1.9) : (m == 2 ? 3.6 : 5.2);
            const double t = (double)waves * (5.0 + tile * (double)tiles_each) + (s > 1 ? 1.0 : 0.0);
            if (!mt || t < best) { mt = m; splits = s; best = t; }
        }
    }
    if (g_form != 1 && cmlb200_attention_latent_tc_fits(a)) {
        int s = 1;
        const double t = cmlb200_attention_latent_tc_estimate_(a, items, most, keys, &s);
        if (!mt || t < best || g_form == 2)
            return cmlb200_attention_latent_tc_(a, d_q_f16, (long)q_rows * a->heads, d_row_pos, d_row_slot, s, d_tiles, items, most, d_tiles ? rows : 0, d_o_bf16,
                                                as_stream(stream));
    }
    CMLB_REQUIRE(mt > 0, "%s: rank %d and %d elements per token do not fit shared memory", who, a->rank, a->ld);
    const size_t smem = latent_smem(16 * mt, a->ld, rank16 + 4);
    const long per = blocks(mt) / items;
    CMLB_REQUIRE(per <= 65535, "%s: %d heads", who, a->heads);
    const dim3 grid(splits, (unsigned)per, items);
    static size_t attr[9][kMaxDevices] = {};
    cudaStream_t st = as_stream(stream);
#define LT_LAUNCH(MT, CU, slot)                                                                                                  \
    do {                                                                                                                         \
        auto kern = attention_latent_kernel<MT, CU>;                                                                             \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                     \
        if (splits > 8) CMLB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));                \
        CMLB_CUDA(launch_chain(kern, grid, dim3(LT_THREADS), smem, splits, st, *a, (const __half*)d_q_f16, d_row_pos, d_row_slot, (const int4*)d_tiles, d_tiles ? rows : 0, \
                               (__nv_bfloat16*)d_o_bf16));                                                                       \
    } while (0)
#define LT_RANK(MT, slot)                                     \
    do {                                                      \
        if (rank16 <= 128) LT_LAUNCH(MT, 1, slot);            \
        else if (rank16 <= 256) LT_LAUNCH(MT, 2, slot + 1);   \
        else LT_LAUNCH(MT, 4, slot + 2);                      \
    } while (0)
    if (mt == 1) LT_RANK(1, 0);
    else if (mt == 2) LT_RANK(2, 3);
    else LT_RANK(4, 6);
#undef LT_RANK
#undef LT_LAUNCH
    return CMLB200_OK;
}
