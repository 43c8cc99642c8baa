// Attention over latents on the 5th-generation tensor cores: the same operation as attention_latent.cu, for latents
// whose operands fit shared memory.
//
// A CTA holds up to 32 or 64 (token, head) rows of queries and walks key tiles of 64 tokens; a cluster of up to 8 CTAs
// (4 for 64 rows) splits the tiles and merges through distributed shared memory. Latents of more than 256 values give two CTAs a half
// of the output columns each (both compute the scores). Roles:
//   warps 0, 2, 3  TMA: the queries once, then key tiles, 16 tokens to a copy (the block table says where), in slabs of 64
//              columns with 128-byte swizzle; the slabs are shared out, since issuing the many small copies takes long.
//              Slabs that are values too stay until O has taken them and have two or three stages, the others are free
//              after the scores and have two
//   warp 1     owns tensor memory; issues tcgen05.mma: S = Q K^T into two alternating accumulators, and
//              O += P V, where V is the same tile read with its columns as the contiguous dimension; whichever of the two
//              has its operands goes first
//   warps 4, 5 softmax, a thread per row (warp 5 for 64 rows): S from tensor memory, mask, exponentials, P as fp16
//              into shared memory. The reference of the exponentials moves, and O is scaled, only when a row's maximum has grown by more than 8 (a factor of 256); sums are fp32
// The scores of tile i + 1 are computed while the softmax of tile i runs. An MMA is 128 rows high: those past the CTA's
// read whatever follows in shared memory and are never looked at. Keys past the sequence's last are zeroed in the tile,
// so that nothing other requests left in a block can reach the sums.
// Every wait is bounded; one that gives up leaves a code in a status word in host memory, and the CTA still drains its
// copies, meets its cluster and frees its tensor memory.
#include "tcgen05_util.cuh"

namespace {

constexpr int TC_THREADS = 192, TC_LOADERS = 3, TC_KEYS = 64, TC_SLAB = TC_KEYS * 128, TC_S_COL = 256, TC_TMEM = 512;

// Slabs of a tile: `v` of them are values of this launch's CTAs too (`stages` copies), `k` are keys alone (two copies).
struct TcSlabs {
    int all, v, k, stages;
};
__host__ __device__ inline size_t tc_operands(int mr, const TcSlabs& t) { return (size_t)t.all * mr * 128 + (size_t)mr * 128 + (size_t)(t.stages * t.v + 2 * t.k) * TC_SLAB; }
__host__ __device__ constexpr int tc_splits(int mr) { return mr == 32 ? 8 : 4; }
__host__ __device__ inline size_t tc_smem(int mr, const TcSlabs& t) { return tc_operands(mr, t) + 256 + 2 * 4 * (size_t)tc_splits(mr) * mr; }

// grid = (splits, row blocks * halves, items), clusters of `splits` CTAs along x.
template <int MR>
__global__ void __launch_bounds__(TC_THREADS, 1)
attention_latent_tc_kernel(const __grid_constant__ CUtensorMap qmap, const __grid_constant__ CUtensorMap kmap, const cmlb200_latent a,
                           const int* __restrict__ row_pos, const int* __restrict__ row_slot, const int4* __restrict__ tiles, int first,
                           __nv_bfloat16* __restrict__ out, int halves, const TcSlabs sl, int* status) {
    extern __shared__ __align__(1024) uint8_t smem[];
    constexpr int TC_SPLITS = tc_splits(MR);
    if (smem_addr(smem) & 1023) {                                       // the swizzle needs it; the declaration asks for it
        if (threadIdx.x == 0) *(volatile int*)status = 9;
        return;
    }
    const int v_bytes = sl.v * TC_SLAB, k_bytes = sl.k * TC_SLAB;
    const uint32_t qs = smem_addr(smem), ps = qs + sl.all * MR * 128, vs = ps + MR * 128, ks = vs + sl.stages * v_bytes;
    uint8_t* tail = smem + tc_operands(MR, sl);
    const uint32_t bars = smem_addr(tail);
    const uint32_t q_full = bars, p_full = bars + 8, pv_done = bars + 16;
    auto s_full = [&](int s) { return bars + 24 + 8 * s; };
    auto k_full = [&](int s) { return bars + 40 + 8 * s; };
    auto k_empty = [&](int s) { return bars + 56 + 8 * s; };
    auto v_full = [&](int s) { return bars + 72 + 8 * s; };
    auto v_empty = [&](int s) { return bars + 96 + 8 * s; };
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(tail + 128);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tail + 136);
    float* c_m = reinterpret_cast<float*>(tail + 256);
    float* c_l = c_m + TC_SPLITS * MR;                                  // [TC_SPLITS][MR] maxima and sums of the whole cluster
    float* Os = reinterpret_cast<float*>(smem);                         // [MR][columns + 4], over the operands once they are done
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        mbar_init(p_full, MR / 32);
        mbar_init(pv_done, 1);
        for (int s = 0; s < 2; s++) { mbar_init(k_full(s), TC_LOADERS); mbar_init(k_empty(s), 1); mbar_init(s_full(s), 1); }
        for (int s = 0; s < 3; s++) { mbar_init(v_full(s), TC_LOADERS); mbar_init(v_empty(s), 1); }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_addr(tmem_slot)), "r"((uint32_t)TC_TMEM) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tmem_fence_before();
    __syncthreads();
    tmem_fence_after();
    const uint32_t tmem = *tmem_slot;
    // a launch that allocates tensor memory too may start from here on: every CTA of this one has its own
    dep_wait();
    dep_trigger();

    // first phase of the cluster's barrier: nothing is stored into another CTA before that one runs
    if (gridDim.x > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
    int4 tl = tiles ? tiles[blockIdx.z] : make_int4((int)blockIdx.z, 1, row_slot[blockIdx.z], row_pos[blockIdx.z]);
    tl.x -= first;
    const int total = tl.y * a.heads, half = blockIdx.y % halves, m0 = blockIdx.y / halves * MR;
    const bool live = m0 < total;                                       // the same for a whole cluster
    const int splits = gridDim.x, rank = blockIdx.x, shift = __ffs(a.block_size) - 1;
    const int* table = a.block_table + (size_t)tl.z * a.table_ld;
    const int window = a.window > 0 ? a.window : 0x7fffffff;
    const int p_first = tl.w + m0 / a.heads, p_last = tl.w + (min(m0 + MR, total) - 1) / a.heads;
    const int k_lo = (window > p_first ? 0 : p_first - window + 1) & ~15;
    const int ntiles = live ? (p_last - k_lo) / TC_KEYS + 1 : 0;
    const int n = rank < ntiles ? (ntiles - rank + splits - 1) / splits : 0;          // tiles of this CTA: rank, rank + splits, ..
    // slabs v0 .. v0 + sl.v - 1 are this half's values; of an odd number both halves take the middle one
    const int nv = (a.rank + 63) / 64, v0 = half * (nv - sl.v), cols = sl.v * 64;
    const int row0 = tl.x * a.heads + m0;

    if (warp == 0 || warp == 2 || warp == 3) {
        const int w = warp ? warp - 1 : 0;                              // slabs w, w + 3, .. of either kind
        bool ok = true;
        int i = 0, vst = 0, vpar = 1;
        if (n > 0 && w == 0) {
            if (elect_one()) {
                mbar_expect_tx(q_full, (uint32_t)(sl.all * MR * 128));
                for (int s = 0; s < sl.all; s++) tma_load_2d(qs + s * MR * 128, &qmap, s * 64, row0, q_full);
            }
            __syncwarp();
        }
        // this warp's share of `count` slabs, the tile's slabs from `from` on (`skip` of them left out behind `gap`)
        auto load = [&](const int (&slot)[4], int count, int from, int gap, int skip, uint32_t dst, uint32_t bar) {
            const int mine = (count - w + TC_LOADERS - 1) / TC_LOADERS;
            if (elect_one()) {
                mbar_expect_tx(bar, (uint32_t)(max(mine, 0) * TC_SLAB));
                for (int c = w; c < count; c += TC_LOADERS) {
                    const int x = (from + c + (c >= gap ? skip : 0)) * 64;
#pragma unroll
                    for (int g = 0; g < 4; g++) tma_load_2d(dst + c * TC_SLAB + g * 2048, &kmap, x, slot[g], bar);
                }
            }
            __syncwarp();
        };
        for (; i < n; i++) {
            const int kt = k_lo + (rank + i * splits) * TC_KEYS;
            // where the four blocks of 16 tokens lie; past the end the last one again
            const int key = min(kt + 16 * (lane & 3), p_last & ~15), at = (table[key >> shift] << shift) + (key & (a.block_size - 1));
            const int slot[4] = {__shfl_sync(0xffffffffu, at, 0), __shfl_sync(0xffffffffu, at, 1), __shfl_sync(0xffffffffu, at, 2), __shfl_sync(0xffffffffu, at, 3)};
            if (sl.k) {
                ok = __all_sync(0xffffffffu, mbar_wait(k_empty(i & 1), ((i >> 1) & 1) ^ 1, abort_flag, 1, status));
                if (!ok) break;
                load(slot, sl.k, 0, v0, sl.v, ks + (i & 1) * k_bytes, k_full(i & 1));
            }
            ok = __all_sync(0xffffffffu, mbar_wait(v_empty(vst), vpar, abort_flag, 1, status));
            if (!ok) break;
            load(slot, sl.v, v0, sl.v, 0, vs + vst * v_bytes, v_full(vst));
            if (++vst == sl.stages) { vst = 0; vpar ^= 1; }
        }
        if (!ok && n > 0) {                                             // no copy outlives the CTA: tiles 0 .. i - 1, and the keys of tile i
            if (w == 0) mbar_wait(q_full, 0, abort_flag, 2, status);
            for (int j = max(0, i - sl.stages); j < i; j++) mbar_wait(v_full(j % sl.stages), (j / sl.stages) & 1, abort_flag, 2, status);
            for (int j = max(0, i - 1); j <= i && sl.k; j++)
                for (uint32_t it = 0; it < 65536 && !mbar_test(k_full(j & 1), (j >> 1) & 1); it++) __nanosleep(32);
        }
    } else if (warp == 1) {
        if (n > 0) {
            // fp16 operands, fp32 accumulators, 128 rows; the second one takes V with its columns contiguous
            const uint32_t is = (1u << 4) | ((uint32_t)(TC_KEYS >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
            const uint32_t io = (1u << 4) | (1u << 16) | ((uint32_t)(cols >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
            const uint32_t acc = __shfl_sync(0xffffffffu, tmem, 0);
            const int last = (a.ld & 63) >> 4;                          // steps of 16 columns in the last slab, 0: all four
            bool ok = __all_sync(0xffffffffu, mbar_wait(q_full, 0, abort_flag, 3, status));
            int i_s = 0, i_o = 0, s_st = 0, s_par = 0, o_st = 0;        // next tile of either product, value stages
            uint32_t spins = 0;
            while (ok && i_o < n) {
                bool did = false;
                // at most one tile ahead: the scores of the one before last have been read
                if (i_s < n && i_s <= i_o + 1 && __all_sync(0xffffffffu, mbar_test(v_full(s_st), s_par) && (!sl.k || mbar_test(k_full(i_s & 1), (i_s >> 1) & 1)))) {
                    tmem_fence_after();
                    const uint32_t d = acc + TC_S_COL + (i_s & 1) * TC_KEYS, vst = vs + s_st * v_bytes, kst = ks + (i_s & 1) * k_bytes;
                    // slabs s .. end - 1, which lie one behind the other from `at` on
                    auto run = [&](int s, int end, uint32_t at) {
                        const int whole = end == sl.all && last ? end - 1 : end;
                        uint64_t ad = make_desc(qs + s * MR * 128), bd = make_desc(at);
                        for (; s < whole; s++, ad += (uint64_t)(MR * 128 >> 4), bd += (uint64_t)(TC_SLAB >> 4)) {
                            if (elect_one()) {
#pragma unroll
                                for (int k = 0; k < 4; k++) umma(d, ad + (uint64_t)(2 * k), bd + (uint64_t)(2 * k), is, (s | k) ? 1u : 0u);
                            }
                            __syncwarp();
                        }
                        if (s < end && elect_one()) {
#pragma unroll
                            for (int k = 0; k < 3; k++)
                                if (k < last) umma(d, ad + (uint64_t)(2 * k), bd + (uint64_t)(2 * k), is, (s | k) ? 1u : 0u);
                        }
                        __syncwarp();
                    };
                    run(0, v0, kst);
                    run(v0, v0 + sl.v, vst);
                    run(v0 + sl.v, sl.all, kst + v0 * TC_SLAB);
                    if (elect_one()) {
                        if (sl.k) umma_commit(k_empty(i_s & 1));
                        umma_commit(s_full(i_s & 1));
                    }
                    __syncwarp();
                    if (++s_st == sl.stages) { s_st = 0; s_par ^= 1; }
                    i_s++;
                    did = true;
                }
                if (i_o < i_s && __all_sync(0xffffffffu, mbar_test(p_full, i_o & 1))) {
                    tmem_fence_after();
                    const uint64_t pd = make_desc(ps), vd = make_desc_mn(vs + o_st * v_bytes, TC_SLAB);
                    if (elect_one()) {
#pragma unroll
                        for (int k = 0; k < TC_KEYS / 16; k++) umma(acc, pd + (uint64_t)(2 * k), vd + (uint64_t)(k * (2048 >> 4)), io, (i_o | k) ? 1u : 0u);
                        umma_commit(v_empty(o_st));
                        umma_commit(pv_done);
                    }
                    __syncwarp();
                    if (++o_st == sl.stages) o_st = 0;
                    i_o++;
                    did = true;
                }
                if (did) {
                    spins = 0;
                } else if (++spins > 1024) {
                    ok = !__any_sync(0xffffffffu, *abort_flag != 0);
                    __nanosleep(32);
                    if (ok && spins > SPIN_LIMIT) {
                        ok = false;
                        *abort_flag = 4;
                        if (*(volatile int*)status == 0) *(volatile int*)status = 4;
                    }
                }
            }
        }
        __syncwarp();
    } else if (warp >= 4 && (warp & 3) * 32 < MR && live) {
        const int q = warp & 3, r = q * 32 + lane;                      // the quarter of tensor memory's lanes this warp may read
        const uint32_t lanes = tmem + ((uint32_t)(q * 32) << 16);
        const int p = m0 + r < total ? tl.w + (m0 + r) / a.heads : -1;
        float m = -INFINITY, l = 0.f;
        bool ok = true;
        int vst = 0;
        for (int i = 0; i < n; i++, vst = vst + 1 == sl.stages ? 0 : vst + 1) {
            const int kt = k_lo + (rank + i * splits) * TC_KEYS;
            ok = __all_sync(0xffffffffu, mbar_wait(s_full(i & 1), (i >> 1) & 1, abort_flag, 6, status));
            if (!ok) break;
            tmem_fence_after();
            uint32_t v[2][32];
            tmem_ld32(lanes + TC_S_COL + (i & 1) * TC_KEYS, v[0]);
            tmem_ld32(lanes + TC_S_COL + (i & 1) * TC_KEYS + 32, v[1]);
            if (kt + TC_KEYS - 1 > p_first || kt <= p_last - window) {
#pragma unroll
                for (int j = 0; j < TC_KEYS; j++) {
                    const int d = p - kt - j;
                    if (d < 0 || d >= window) v[j >> 5][j & 31] = 0xff800000u;
                }
            }
            float mx = -INFINITY;
#pragma unroll
            for (int j = 0; j < TC_KEYS; j++) mx = fmaxf(mx, __uint_as_float(v[j >> 5][j & 31]));
            float c = 1.f;
            const bool scale = __any_sync(0xffffffffu, mx > m + 8.f);  // -inf + 8 is -inf: a row's first keys count
            if (scale) {
                const float nm = fmaxf(m, mx);
                c = nm == -INFINITY ? 1.f : ex2(m - nm);
                m = nm;
                l *= c;
            }
            const float u = m == -INFINITY ? 0.f : m;
            uint32_t pk[TC_KEYS / 2];
            float l2 = 0.f;
#pragma unroll
            for (int j = 0; j < TC_KEYS / 2; j++) {
                const float e0 = ex2(__uint_as_float(v[j >> 4][(2 * j) & 31]) - u), e1 = ex2(__uint_as_float(v[j >> 4][(2 * j + 1) & 31]) - u);
                l += e0;
                l2 += e1;
                const __half2 h = __floats2half2_rn(e0, e1);
                pk[j] = *reinterpret_cast<const uint32_t*>(&h);
            }
            l += l2;
            if (i > 0) {                                                // P and O are the last product's until it is done
                ok = __all_sync(0xffffffffu, mbar_wait(pv_done, (i - 1) & 1, abort_flag, 7, status));
                if (!ok) break;
                tmem_fence_after();
                if (scale) {
                    for (int c0 = 0; c0 < cols; c0 += 32) {
                        uint32_t o[32];
                        tmem_ld32(lanes + c0, o);
#pragma unroll
                        for (int j = 0; j < 32; j++) o[j] = __float_as_uint(__uint_as_float(o[j]) * c);
                        tmem_st32(lanes + c0, o);
                    }
                    tmem_st_wait();
                }
            }
            uint8_t* prow = smem + (ps - qs) + r * 128;
#pragma unroll
            for (int j = 0; j < 8; j++) *reinterpret_cast<uint4*>(prow + ((j ^ (r & 7)) << 4)) = make_uint4(pk[4 * j], pk[4 * j + 1], pk[4 * j + 2], pk[4 * j + 3]);
            const int valid = p_last - kt + 1;                          // keys of this tile that exist
            if (valid < TC_KEYS) {
                uint8_t* v = smem + (vs - qs) + vst * v_bytes;
                const int chunks = (TC_KEYS - valid) * 8;
                for (int j = r; j < chunks * sl.v; j += MR)
                    *reinterpret_cast<uint4*>(v + j / chunks * TC_SLAB + valid * 128 + j % chunks * 16) = make_uint4(0u, 0u, 0u, 0u);
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            tmem_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full);
        }
        if (ok && n > 0) ok = __all_sync(0xffffffffu, mbar_wait(pv_done, (n - 1) & 1, abort_flag, 8, status));
        tmem_fence_after();
        if (!ok) { m = -INFINITY; l = 0.f; }
        __syncwarp();
        if (splits > 1) {
            asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
#pragma unroll
            for (int s = 0; s < TC_SPLITS; s++) {
                if (s < splits) {
                    uint32_t am, al;
                    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(am) : "r"(smem_addr(c_m + rank * MR + r)), "r"(s));
                    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(al) : "r"(smem_addr(c_l + rank * MR + r)), "r"(s));
                    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(am), "f"(m) : "memory");
                    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(al), "f"(l) : "memory");
                }
            }
        }
        // a sink carries no value; with several splits it joins below
        const float all = l > 0.f && a.sinks && splits == 1 ? l + exp2f(a.sinks[(m0 + r) % a.heads] * kLog2e - m) : l;
        const float inv = all > 0.f ? 1.0f / all : 0.f;
        for (int c0 = 0; c0 < cols && n > 0; c0 += 32) {
            uint32_t o[32];
            tmem_ld32(lanes + c0, o);
            if (splits > 1) {
                float4* d = reinterpret_cast<float4*>(Os + r * (cols + 4) + c0);
#pragma unroll
                for (int j = 0; j < 8; j++)
                    d[j] = make_float4(__uint_as_float(o[4 * j]), __uint_as_float(o[4 * j + 1]), __uint_as_float(o[4 * j + 2]), __uint_as_float(o[4 * j + 3]));
            } else if (m0 + r < total) {
                uint32_t w[16];
#pragma unroll
                for (int j = 0; j < 16; j++) {
                    const int col = v0 * 64 + c0 + 2 * j;
                    const __nv_bfloat162 h = __floats2bfloat162_rn(col < a.rank ? __uint_as_float(o[2 * j]) * inv : 0.f, col + 1 < a.rank ? __uint_as_float(o[2 * j + 1]) * inv : 0.f);
                    w[j] = *reinterpret_cast<const uint32_t*>(&h);
                }
                uint4* d = reinterpret_cast<uint4*>(out + (size_t)(row0 + r) * a.ld_rank + v0 * 64 + c0);
#pragma unroll
                for (int j = 0; j < 4; j++) d[j] = make_uint4(w[4 * j], w[4 * j + 1], w[4 * j + 2], w[4 * j + 3]);
            }
        }
        tmem_fence_before();
    }
    __syncwarp();
    if (splits > 1 && !(warp >= 4 && (warp & 3) * 32 < MR && live)) asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    if (splits > 1 && live) {
        asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
        asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
        const int rows = min(MR, total - m0), quads = cols / 4;
        for (int i = rank * TC_THREADS + threadIdx.x; i < rows * quads; i += splits * TC_THREADS) {
            const int r = i / quads, c = (i - r * quads) * 4;
            float4 xs[TC_SPLITS];
#pragma unroll
            for (int s = 0; s < TC_SPLITS; s++) {
                xs[s] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (s < splits) {
                    uint32_t ax;
                    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(ax) : "r"(smem_addr(Os + r * (cols + 4) + c)), "r"(s));
                    asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(xs[s].x), "=f"(xs[s].y), "=f"(xs[s].z), "=f"(xs[s].w) : "r"(ax) : "memory");
                }
            }
            float mx = -INFINITY, sum = 0.f;
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int s = 0; s < TC_SPLITS; s++) mx = fmaxf(mx, s < splits ? c_m[s * MR + r] : -INFINITY);
#pragma unroll
            for (int s = 0; s < TC_SPLITS; s++) {
                if (s >= splits || c_m[s * MR + r] == -INFINITY) continue;      // saw nothing: its values may be anything
                const float f = exp2f(c_m[s * MR + r] - mx);
                sum = fmaf(c_l[s * MR + r], f, sum);
                x.x = fmaf(xs[s].x, f, x.x); x.y = fmaf(xs[s].y, f, x.y); x.z = fmaf(xs[s].z, f, x.z); x.w = fmaf(xs[s].w, f, x.w);
            }
            if (a.sinks && sum > 0.f) sum += exp2f(a.sinks[(m0 + r) % a.heads] * kLog2e - mx);
            const float inv = sum > 0.f ? 1.0f / sum : 0.f;
            const int col = v0 * 64 + c;
            const __nv_bfloat162 lo = __floats2bfloat162_rn(col < a.rank ? x.x * inv : 0.f, col + 1 < a.rank ? x.y * inv : 0.f);
            const __nv_bfloat162 hi = __floats2bfloat162_rn(col + 2 < a.rank ? x.z * inv : 0.f, col + 3 < a.rank ? x.w * inv : 0.f);
            *reinterpret_cast<uint2*>(out + (size_t)(row0 + r) * a.ld_rank + col) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        }
        asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");  // nobody leaves while others read its shared memory
        asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    }
    tmem_fence_before();
    __syncthreads();
    if (warp == 1) {
        tmem_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"((uint32_t)TC_TMEM) : "memory");
    }
}

int* g_status[kMaxDevices] = {};

int status_word(int** word) {
    int dev = 0;
    CMLB_CUDA(cudaGetDevice(&dev));
    CMLB_REQUIRE(dev >= 0 && dev < kMaxDevices, "device %d", dev);
    if (!g_status[dev]) {
        void* p = nullptr;
        CMLB_CUDA(cudaHostAlloc(&p, sizeof(int), cudaHostAllocDefault));
        *static_cast<int*>(p) = 0;
        g_status[dev] = static_cast<int*>(p);
    }
    *word = g_status[dev];
    return CMLB200_OK;
}

}  // namespace

// Slabs and stages for CTAs of mr rows; stages 0: the operands do not fit.
static TcSlabs tc_plan(const cmlb200_latent* a, int mr) {
    TcSlabs t;
    t.all = (a->ld + 63) / 64;
    t.v = a->rank > 256 ? (a->rank + 127) / 128 : (a->rank + 63) / 64;
    t.k = t.all - t.v;
    for (t.stages = 3; t.stages > 1 && tc_smem(mr, t) > 227 * 1024; t.stages--) {}
    if (t.stages == 1) t.stages = 0;
    return t;
}

// One CTA to an SM: each needs all of the SM's tensor memory, and a cluster's CTAs wait for one another.
static size_t tc_bytes(int mr, const TcSlabs& sl) {
    const size_t need = tc_smem(mr, sl);
    return need > 118 * 1024 ? need : 118 * 1024;
}

// 1: these sizes run here. Operands must fit, and the pool's extent must be known for its tensor map.
extern "C" int cmlb200_attention_latent_tc_fits(const cmlb200_latent* a) { return a && a->pool_blocks > 0 && a->rank > 0 && a->rank <= 512 && a->ld <= 2048 && tc_plan(a, 64).stages > 0; }

// CTAs that run at a time when clusters of `splits` share the device: one to an SM, and a cluster stays within a group of
// SMs whose size it may not divide.
static long tc_room(int mr, int splits, size_t smem) {
    static int active[2][4][kMaxDevices] = {};
    if (splits == 1) return cmlb_num_sms();
    int* n = &active[mr == 64][splits == 2 ? 1 : (splits == 4 ? 2 : 3)][cmlb_device_index()];
    if (!*n) {
        cudaLaunchAttribute attr;
        attr.id = cudaLaunchAttributeClusterDimension;
        attr.val.clusterDim.x = (unsigned)splits;
        attr.val.clusterDim.y = attr.val.clusterDim.z = 1;
        cudaLaunchConfig_t cfg = {};
        cfg.gridDim = dim3(splits);
        cfg.blockDim = dim3(TC_THREADS);
        cfg.dynamicSmemBytes = smem;
        cfg.attrs = &attr;
        cfg.numAttrs = 1;
        const void* kern = mr == 32 ? (const void*)attention_latent_tc_kernel<32> : (const void*)attention_latent_tc_kernel<64>;
        if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess ||
            cudaOccupancyMaxActiveClusters(n, kern, &cfg) != cudaSuccess || *n < 1) {
            cudaGetLastError();
            *n = cmlb_num_sms() / splits * 3 / 4;
        }
    }
    return (long)*n * splits;
}

// Microseconds, by estimate, of the best split of the keys.
extern "C" double cmlb200_attention_latent_tc_estimate_(const cmlb200_latent* a, int items, int most, int keys, int* splits) {
    const int mr = most <= 32 ? 32 : 64;
    const size_t smem = tc_bytes(mr, tc_plan(a, mr));
    const long blocks = (long)items * ((most + mr - 1) / mr) * (a->rank > 256 ? 2 : 1);
    double best = 0.0;
    for (int s = 1; s <= tc_splits(mr) && (s == 1 || (s - 1) * TC_KEYS < keys); s *= 2) {
        const long ctas = blocks * s, room = tc_room(mr, s, smem), waves = (ctas + room - 1) / room, each = ((keys + TC_KEYS - 1) / TC_KEYS + s - 1) / s;
        const double t = (double)waves * (9.0 + 1.8 * (double)each) + (s > 1 ? 2.0 : 0.0);
        if (s == 1 || t < best) { *splits = s; best = t; }
    }
    return best;
}

extern "C" int cmlb200_attention_latent_tc_(const cmlb200_latent* a, const uint16_t* q, long q_rows, const int* row_pos, const int* row_slot, int splits,
                                            const int* tiles, int items, int most, int first, uint16_t* o, cudaStream_t st) {
    const int mr = most <= 32 ? 32 : 64, halves = a->rank > 256 ? 2 : 1;
    const long blocks = (long)((most + mr - 1) / mr) * halves;
    CMLB_REQUIRE(blocks <= 65535, "cmlb200_attention_latent: %d heads", a->heads);
    int* status;
    int rc = status_word(&status);
    if (rc) return rc;
    CUtensorMap qmap, kmap;
    rc = encode_map(&qmap, CU_TENSOR_MAP_DATA_TYPE_FLOAT16, q, q_rows, a->ld, a->ld, 64, mr);
    if (!rc) rc = encode_map(&kmap, CU_TENSOR_MAP_DATA_TYPE_FLOAT16, a->pool, (long)a->pool_blocks * a->block_size, a->ld, a->ld, 64, 16);
    if (rc) return rc;
    const TcSlabs sl = tc_plan(a, mr);
    const size_t smem = tc_bytes(mr, sl);
    const dim3 grid(splits, (unsigned)blocks, items);
    static size_t attr[2][kMaxDevices] = {};
#define TC_LAUNCH(MR, slot)                                                                                                      \
    do {                                                                                                                         \
        auto kern = attention_latent_tc_kernel<MR>;                                                                              \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                     \
        CMLB_CUDA(launch_chain(kern, grid, dim3(TC_THREADS), smem, splits, st, qmap, kmap, *a, row_pos, row_slot, (const int4*)tiles, first, (__nv_bfloat16*)o, \
                               halves, sl, status));                                                                                 \
    } while (0)
    if (mr == 32) TC_LAUNCH(32, 0);
    else TC_LAUNCH(64, 1);
#undef TC_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_attention_latent_status(int* status, int reset) {
    CMLB_REQUIRE(status, "cmlb200_attention_latent_status: NULL argument");
    int* word;
    const int rc = status_word(&word);
    if (rc) return rc;
    *status = *static_cast<volatile int*>(word);
    if (reset) *static_cast<volatile int*>(word) = 0;
    return CMLB200_OK;
}
