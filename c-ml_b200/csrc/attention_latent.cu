// Attention over latents: every head of a row attends the same keys, one vector [latent | rotated part] per token of a
// paged cache, and the weighted sum of the latents is what a head returns. Queries come transformed
// (cmlb200_latent_query), in units of log2. One kernel serves decoded tokens and short prompt portions:
// the (token, head) pairs of a portion are the rows of the matrix products, 16, 32 or 64 to a CTA.
//
// A key tile of 32 tokens is fetched once through the block table (cp.async, three stages) and serves both products on
// mma.sync m16n8k16: S = Q K^T with the warps splitting rows, keys and, for few rows, the key columns; O += P K with the
// warps splitting the latent's columns. Scores pass through shared memory, where a few threads per row keep
// the running maximum and sum in fp32. A cluster of up to 8 CTAs splits the keys and merges through distributed
// shared memory, each CTA finishing a share of the values.
#include "lm_util.cuh"

namespace {

constexpr int LT_THREADS = 256, LT_WARPS = 8, LT_KEYS = 32, LT_STAGES = 3, LT_SLD = LT_KEYS + 4, LT_PLD = LT_KEYS + 8;

__host__ __device__ inline size_t latent_smem(int rows, int ld, int ldo) {
    const size_t lk = ld + 8;
    const size_t tiles = 2 * lk * (rows + LT_STAGES * LT_KEYS), merge = 4 * (size_t)rows * ldo;
    // operands, or the merged values in their place; scores (64 rows of partial sums), weights, per-row factors
    return (tiles > merge ? tiles : merge) + 4 * 64 * LT_SLD + 2 * (size_t)rows * LT_PLD + 3 * 4 * (size_t)rows;
}

// grid = (splits, ceil(tokens * heads / (16 MT)), items), clusters of `splits` CTAs along x. CU: 16-column groups of the
// latent per warp.
template <int MT, int CU>
__global__ void __launch_bounds__(LT_THREADS)
attention_latent_kernel(const cmlb200_latent a, const __half* __restrict__ q, const int* __restrict__ row_pos, const int* __restrict__ row_slot,
                        const int4* __restrict__ tiles, int first, __nv_bfloat16* __restrict__ out) {
    constexpr int MR = 16 * MT, KS = 4 / MT, TPR = LT_THREADS / MR, KPT = LT_KEYS / TPR;
    extern __shared__ __align__(16) uint8_t sm[];
    const int LK = a.ld + 8, rank16 = (a.rank + 15) & ~15, LDO = rank16 + 4;
    __half* Qs = reinterpret_cast<__half*>(sm);
    __half* Ks = Qs + MR * LK;
    const size_t tile_bytes = 2 * (size_t)LK * (MR + LT_STAGES * LT_KEYS), merge_bytes = 4 * (size_t)MR * LDO;
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

    auto load = [&](int it, int stage) {
        if (it < ntiles) {
            const int row = threadIdx.x >> 3, key = min(k_lo + it * LT_KEYS + row, p_last);       // past the end: the last key, masked below
            const __half* src = pool + (((size_t)table[key >> shift] << shift) + (key & (a.block_size - 1))) * a.ld;
            const uint32_t dst = smem_addr(Ks + (stage * LT_KEYS + row) * LK);
            for (int c = threadIdx.x & 7; c < kc; c += 8) cp16(dst + c * 16, src + c * 8);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    {
        const __half* src = q + ((size_t)tl.x * a.heads + m0) * a.ld;
        for (int i = threadIdx.x; i < MR * kc; i += LT_THREADS) {
            const int r = i / kc, c = i - r * kc;
            cp16(smem_addr(Qs + r * LK + c * 8), src + (size_t)min(r, total - 1 - m0) * a.ld + c * 8);
        }
    }
    load(rank, 0);
    load(rank + splits, 1);

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
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();                                                // this tile is there; the stage of the one before is free
        load(it + 2 * splits, stage == 0 ? 2 : stage - 1);
        {
            float s[2][4] = {};
            const uint32_t k_base = smem_addr(Ks + (stage * LT_KEYS + w_k * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * LK + ((lane >> 3) & 1) * 8);
#pragma unroll 4
            for (int kk = w_s * 16; kk < a.ld; kk += KS * 16) {
                uint32_t qa[4], b[4];
                ldsm4(q_base + kk * 2, qa);
                ldsm4(k_base + kk * 2, b);
                mma_f16(s[0], qa, b[0], b[1]);
                mma_f16(s[1], qa, b[2], b[3]);
            }
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
#pragma unroll
            for (int u = 0; u < CU; u++) {
                const int col = (u * LT_WARPS + warp) * 16;
                if (col < rank16) {
#pragma unroll
                    for (int kk = 0; kk < LT_KEYS / 16; kk++) {
                        uint32_t b[4];
                        ldsm4_t(v_base + (kk * 16 * LK + col) * 2, b);
#pragma unroll
                        for (int i = 0; i < MT; i++) {
                            mma_f16(o[i][u][0], pa[i][kk], b[0], b[1]);
                            mma_f16(o[i][u][1], pa[i][kk], b[2], b[3]);
                        }
                    }
                }
            }
        }
        stage = stage == 2 ? 0 : stage + 1;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int w = 1; w < TPR; w <<= 1) l += __shfl_xor_sync(0xffffffffu, l, w);
    __syncthreads();                                                    // every warp is done with the operands and `corr`
    if (sk == 0) {
        c_m[sr] = m;
        c_l[sr] = l;
        corr[sr] = l > 0.f ? 1.0f / l : 0.f;
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
    const int live = min(MR, total - m0);
    for (int i = rank * LT_THREADS + threadIdx.x; i < live * a.rank; i += splits * LT_THREADS) {
        const int r = i / a.rank, d = i - r * a.rank;
        float ms[8], ls[8], xs[8];
#pragma unroll
        for (int s = 0; s < 8; s++) {
            ms[s] = -INFINITY; ls[s] = 0.f; xs[s] = 0.f;
            if (s < splits) {
                uint32_t am, al, ax;
                asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(am) : "r"(smem_addr(c_m + r)), "r"(s));
                asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(al) : "r"(smem_addr(c_l + r)), "r"(s));
                asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(ax) : "r"(smem_addr(Os + r * LDO + d)), "r"(s));
                asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(ms[s]) : "r"(am) : "memory");
                asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(ls[s]) : "r"(al) : "memory");
                asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(xs[s]) : "r"(ax) : "memory");
            }
        }
        float mx = ms[0], x = 0.f, sum = 0.f;
#pragma unroll
        for (int s = 1; s < 8; s++) mx = fmaxf(mx, ms[s]);
#pragma unroll
        for (int s = 0; s < 8; s++) {
            const float c = ms[s] == -INFINITY ? 0.f : exp2f(ms[s] - mx);
            x = fmaf(xs[s], c, x);
            sum = fmaf(ls[s], c, sum);
        }
        out[(out0 + r) * a.ld_rank + d] = __float2bfloat16_rn(x / sum);
    }
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");      // nobody leaves while others read its shared memory
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}

}  // namespace

extern "C" int cmlb200_attention_latent(const cmlb200_latent* a, const uint16_t* d_q_f16, const int* d_row_pos, const int* d_row_slot, int rows, int max_keys,
                                        const int* d_tiles, int tiles, uint16_t* d_o_bf16, void* stream) {
    static const char* who = "cmlb200_attention_latent";
    CMLB_REQUIRE(a && d_q_f16 && d_o_bf16 && (d_tiles ? tiles > 0 && rows >= 0 : d_row_pos && d_row_slot && rows > 0 && max_keys >= 0), "%s: bad argument", who);
    CMLB_REQUIRE(a->heads > 0 && a->rank > 0 && a->ld >= a->rank && a->ld % 16 == 0 && a->ld_rank >= a->rank && a->ld_rank % 64 == 0 && a->rank <= 512,
                 "%s: rank %d (up to 512), strides %d / %d", who, a->rank, a->ld, a->ld_rank);
    CMLB_REQUIRE(a->pool && a->block_table && a->table_ld > 0 && a->cache_dtype == CMLB200_DT_F16, "%s: fp16 cache", who);
    CMLB_REQUIRE(a->block_size >= 16 && (a->block_size & (a->block_size - 1)) == 0, "%s: block size %d must be a power of two >= 16", who, a->block_size);
    CMLB_REQUIRE((((uintptr_t)d_q_f16 | (uintptr_t)a->pool | (uintptr_t)d_tiles) & 15) == 0 && ((uintptr_t)d_o_bf16 & 3) == 0, "%s: alignment", who);
    const int items = d_tiles ? tiles : rows, most = d_tiles ? 64 * a->heads : a->heads, sms = cmlb_num_sms();
    CMLB_REQUIRE(items <= 65535, "%s: %d rows", who, items);
    const int keys = d_tiles ? LT_KEYS : ((a->window > 0 && a->window < max_keys + 1) ? a->window : max_keys + 1);
    const int rank16 = (a->rank + 15) & ~15;
    // rows per CTA: wide tiles read the keys fewest times; narrow ones spread few heads over more SMs
    int mt = most > 32 ? 4 : (most > 16 ? 2 : 1);
    auto blocks = [&](int m) { return (long)items * ((most + 16 * m - 1) / (16 * m)); };
    auto most_splits = [&]() { int s = 1; while (s < 8 && keys > s * LT_KEYS) s *= 2; return s; };
    while (mt > 1 && (latent_smem(16 * mt, a->ld, rank16 + 4) > 227 * 1024 || (!d_tiles && blocks(mt) * most_splits() < sms))) mt /= 2;
    int splits = 1;
    while (splits < 8 && blocks(mt) * splits < sms && keys > splits * LT_KEYS) splits *= 2;
    const size_t smem = latent_smem(16 * mt, a->ld, rank16 + 4);
    CMLB_REQUIRE(smem <= 227 * 1024, "%s: rank %d and %d elements per token do not fit shared memory", who, a->rank, a->ld);
    const long per = blocks(mt) / items;
    CMLB_REQUIRE(per <= 65535, "%s: %d heads", who, a->heads);
    const dim3 grid(splits, (unsigned)per, items);
    static size_t attr[9][kMaxDevices] = {};
    cudaStream_t st = as_stream(stream);
#define LT_LAUNCH(MT, CU, slot)                                                                                                  \
    do {                                                                                                                         \
        auto kern = attention_latent_kernel<MT, CU>;                                                                             \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                     \
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
