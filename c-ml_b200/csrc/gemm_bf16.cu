// Prompt-sized product of dense bf16 weights on the 5th-generation tensor cores:
//   Y[M][N] = X[M][K] W[N][K]^T, bf16 operands, fp32 accumulation in tensor memory.
//
// Persistent: one CTA per SM walks output tiles of 128 rows of x (the MMA "M" side, one per lane of
// tensor memory) by BN weight rows (the "N" side). BN is 256, 128 or 64, picked by how the tiles fill
// the SMs. Roles:
//   warp 0     one lane issues TMA tensor loads of both operands (64-wide K slabs, 128-byte swizzle)
//              into a ring of stages that runs on across tiles
//   warp 1     owns tensor memory; one lane issues tcgen05.mma (128 x BN x 16)
//   warps 2-5  epilogue: tcgen05.ld, through a per-warp transpose buffer to row-contiguous stores
// Two accumulators alternate in tensor memory, so the epilogue of a tile overlaps the next tile's MMAs.
// Output forms: fp32; or the gated activation of weights stored as pairs of 16-row groups (16 gate
// rows, 16 up rows, ...): both halves of a pair sit in one lane's columns, and bf16 act(gate) * up is
// all that leaves the SM; or bf16 act(y); or per-head keys and values as fp16 cache rows. Rows and columns past the edges arrive as
// zeros and are not stored. With a plan of experts the row tiles come from the plan: each has a first row, a number of
// rows and an expert, whose weight rows follow those of the expert before it.
// No cluster multicast. Every mbarrier wait is bounded; on expiry the CTA raises a status word
// (cmlb200_gemm_dense_status), waits for its copies in flight, frees its tensor memory and returns.
#include "tcgen05_util.cuh"

namespace {

constexpr int BM = 128, BK = 64;
constexpr int EPI_WARPS = 4;
constexpr int GEMM_THREADS = 64 + EPI_WARPS * 32;
constexpr int A_BYTES = BM * BK * 2;

template <int BN> struct Tile {
    static constexpr int B_BYTES = BN * BK * 2;
    static constexpr int STAGE = A_BYTES + B_BYTES;
    static constexpr int STAGES = BN == 256 ? 4 : (BN == 128 ? 6 : 8);
    static constexpr int epi_off = STAGES * STAGE;                    // EPI_WARPS x [32][33] fp32
    static constexpr int bar_off = epi_off + EPI_WARPS * 32 * 33 * 4;
    static constexpr int nbars = 2 * STAGES + 4;
    static constexpr int total = bar_off + 8 * nbars + 32;
};

__device__ int g_dense_status = 0;
__device__ __forceinline__ bool mbar_wait(uint32_t bar, uint32_t parity, volatile int* abort_flag, int code) {
    return mbar_wait(bar, parity, abort_flag, code, &g_dense_status);
}

// Tile number -> (row tile, column tile): groups of 8 row tiles share a sweep over the columns, so that
// the CTAs working at one time read few distinct slabs.
__device__ __forceinline__ void tile_at(int i, int tm, int tn, int& m, int& n) {
    const int per = 8 * tn, gq = i / per, in = i - gq * per, rows = min(8, tm - gq * 8);
    m = gq * 8 + in % rows;
    n = in / rows;
}

enum { OUT_F32, OUT_GLU, OUT_ACT, OUT_HEADS };
struct GemmOut {
    int form, act;
    float limit;
    void* y;
    int ldy, n_out;
    const float* bias;                                 // OUT_F32
    float cap;
    // OUT_HEADS: columns below key_cols are heads of `dim` in key rows, those behind them heads of `vdim` in y's rows
    __half* keys;
    int key_cols, dim, dim_ld, vdim, vdim_ld, ldk;
};
struct GemmExperts {
    const int4* tiles;                                 // {first row, expert, rows, 0}; NULL: no experts
    const int* num_tiles;
    int w_rows;
};

template <int BN>
__global__ void __launch_bounds__(GEMM_THREADS, 1)
gemm_bf16_kernel(const __grid_constant__ CUtensorMap xmap, const __grid_constant__ CUtensorMap wmap, int M, int N, int K, const GemmOut out,
                 const GemmExperts ex) {
    using C = Tile<BN>;
    constexpr int ST = C::STAGES;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    const uint32_t sbase = smem_u32(smem), bars = sbase + C::bar_off;
    auto full = [&](int s) { return bars + 8 * s; };
    auto empty = [&](int s) { return bars + 8 * (ST + s); };
    auto acc_full = [&](int b) { return bars + 8 * (2 * ST + b); };
    auto acc_empty = [&](int b) { return bars + 8 * (2 * ST + 2 + b); };
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + C::bar_off + 8 * C::nbars);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + C::bar_off + 8 * C::nbars + 8);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int tn = (N + BN - 1) / BN, nkb = (K + BK - 1) / BK;

    if (threadIdx.x == 0) {
        for (int s = 0; s < ST; s++) { mbar_init(full(s), 1); mbar_init(empty(s), 1); }
        for (int b = 0; b < 2; b++) { mbar_init(acc_full(b), 1); mbar_init(acc_empty(b), EPI_WARPS); }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"((uint32_t)(2 * BN)) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem_base = *tmem_slot;
    dep_wait();
    dep_trigger();
    const int tm = ex.tiles ? *ex.num_tiles : (M + BM - 1) / BM, tiles = tm * tn;

    if (warp == 0) {
        if (lane == 0) {
            int it = 0;
            bool ok = true;
            for (int tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x) {
                int mi, ni;
                tile_at(tile, tm, tn, mi, ni);
                int x0 = mi * BM, w0 = ni * BN;
                if (ex.tiles) { const int4 t = ex.tiles[mi]; x0 = t.x; w0 += t.y * ex.w_rows; }
                for (int k = 0; k < nkb; k++, it++) {
                    const int s = it % ST;
                    ok = mbar_wait(empty(s), ((it / ST) & 1) ^ 1, abort_flag, 1);
                    if (!ok) break;
                    mbar_expect_tx(full(s), (uint32_t)C::STAGE);
                    tma_load_2d(sbase + s * C::STAGE, &xmap, k * BK, x0, full(s));
                    tma_load_2d(sbase + s * C::STAGE + A_BYTES, &wmap, k * BK, w0, full(s));
                }
            }
            for (int i = max(0, it - ST); i < it; i++) mbar_wait(full(i % ST), (i / ST) & 1, abort_flag, 2);      // no copy outlives the CTA
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(BM >> 4) << 24);
            int it = 0, done = 0;
            bool ok = true;
            for (int tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x, done++) {
                const int b = done & 1;
                ok = mbar_wait(acc_empty(b), ((done >> 1) & 1) ^ 1, abort_flag, 3);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                for (int k = 0; k < nkb; k++, it++) {
                    const int s = it % ST;
                    ok = mbar_wait(full(s), (it / ST) & 1, abort_flag, 4);
                    if (!ok) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint64_t ad = make_desc(sbase + s * C::STAGE), bd = make_desc(sbase + s * C::STAGE + A_BYTES);
#pragma unroll
                    for (int kk = 0; kk < BK / 16; kk++)
                        umma(tmem_base + (uint32_t)(b * BN), ad + (uint64_t)(2 * kk), bd + (uint64_t)(2 * kk), idesc, (k | kk) ? 1u : 0u);
                    umma_commit(empty(s));
                }
                umma_commit(acc_full(b));
            }
        }
    } else {
        const int q = warp & 3;                         // the quarter of tensor memory's lanes this warp may read
        float* buf = reinterpret_cast<float*>(smem + C::epi_off) + (warp - 2) * 32 * 33;
        int done = 0;
        for (int tile = blockIdx.x; tile < tiles; tile += gridDim.x, done++) {
            int mi, ni;
            tile_at(tile, tm, tn, mi, ni);
            const int b = done & 1, n0 = ni * BN;
            int m0 = mi * BM + q * 32, m_end = M;
            if (ex.tiles) { const int4 t = ex.tiles[mi]; m0 = t.x + q * 32; m_end = t.x + t.z; }
            const bool ok = __all_sync(0xffffffffu, mbar_wait(acc_full(b), (done >> 1) & 1, abort_flag, 5));
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            for (int c0 = 0; c0 < BN; c0 += 32) {
                uint32_t v[32];
                tmem_ld32(tmem_base + ((uint32_t)(q * 32) << 16) + (uint32_t)(b * BN + c0), v);
                if (c0 + 32 == BN) {                    // this warp has read the whole accumulator
                    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
                    if (lane == 0) mbar_arrive(acc_empty(b));
                }
                if (m0 >= m_end || n0 + c0 >= N) continue;
                __syncwarp();
                if (out.form == OUT_GLU) {
#pragma unroll
                    for (int j = 0; j < 16; j++) buf[lane * 33 + j] = glu_act_fast(out.act, __uint_as_float(v[j]), __uint_as_float(v[16 + j]), out.limit);
                    __syncwarp();
                    const int col = (n0 + c0) / 2 + (lane & 15);
#pragma unroll 4
                    for (int j = 0; j < 32; j += 2) {
                        const int rr = j + (lane >> 4);
                        if (m0 + rr < m_end && col < out.n_out)
                            static_cast<__nv_bfloat16*>(out.y)[(size_t)(m0 + rr) * out.ldy + col] = __float2bfloat16_rn(buf[rr * 33 + (lane & 15)]);
                    }
                } else if (out.form == OUT_ACT) {
                    if (out.act == CMLB200_ACT_GELU_ERF) {      // decided outside, so that the values' chains overlap
#pragma unroll
                        for (int j = 0; j < 32; j++) buf[lane * 33 + j] = gelu_erf_fast(__uint_as_float(v[j]));
                    } else {
#pragma unroll
                        for (int j = 0; j < 32; j++) buf[lane * 33 + j] = unary_act_fast(out.act, __uint_as_float(v[j]));
                    }
                    __syncwarp();
                    const int col = n0 + c0 + 2 * (lane & 15);
#pragma unroll 4
                    for (int j = 0; j < 32; j += 2) {
                        const int rr = j + (lane >> 4);
                        if (m0 + rr >= m_end || col >= out.n_out) continue;
                        const float* s = buf + rr * 33 + 2 * (lane & 15);
                        __nv_bfloat16* d = static_cast<__nv_bfloat16*>(out.y) + (size_t)(m0 + rr) * out.ldy + col;
                        if (col + 1 < out.n_out) *reinterpret_cast<__nv_bfloat162*>(d) = __floats2bfloat162_rn(s[0], s[1]);
                        else *d = __float2bfloat16_rn(s[0]);
                    }
                } else {
#pragma unroll
                    for (int j = 0; j < 32; j++) buf[lane * 33 + j] = __uint_as_float(v[j]);
                    __syncwarp();
                    const int col = n0 + c0 + lane;
                    if (out.form == OUT_F32) {
                        float bias = out.bias && col < out.n_out ? out.bias[col] : 0.f;
                        if (out.cap > 0.f) {
                            for (int j = 0; j < 32; j++) buf[j * 33 + lane] = soft_cap(buf[j * 33 + lane] + bias, out.cap);
                            bias = 0.f;
                        }
#pragma unroll 8
                        for (int j = 0; j < 32; j++)
                            if (m0 + j < m_end && col < out.n_out) static_cast<float*>(out.y)[(size_t)(m0 + j) * out.ldy + col] = buf[j * 33 + lane] + bias;
                    } else {
                        const bool key = col < out.key_cols;
                        const int c = key ? col : col - out.key_cols, per = key ? out.dim : out.vdim, ldo = key ? out.ldk : out.ldy;
                        __half* o = (key ? out.keys : static_cast<__half*>(out.y)) + c / per * (key ? out.dim_ld : out.vdim_ld) + c % per;
#pragma unroll 8
                        for (int j = 0; j < 32; j++)
                            if (m0 + j < m_end && col < out.n_out) o[(size_t)(m0 + j) * ldo] = narrow<__half>(buf[j * 33 + lane]);
                    }
                }
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"((uint32_t)(2 * BN)) : "memory");
    }
}

int make_map(CUtensorMap* map, const void* base, int rows, int cols, int ld, int box_rows) {
    return encode_map(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, base, rows, cols, ld, BK, box_rows);
}

// rows of x and W the maps cover; M: rows of output, or an upper bound of the row tiles times BM
template <int BN>
int launch_gemm(const cmlb200_dense* W, const uint16_t* x, int ldx, int x_rows, int M, int N, const GemmOut& out, const GemmExperts& ex, cudaStream_t st) {
    CUtensorMap xmap, wmap;
    int rc = make_map(&xmap, x, x_rows, W->cols, ldx, BM);
    if (!rc) rc = make_map(&wmap, W->w, W->rows, W->cols, W->ld, BN);
    if (rc) return rc;
    const int tiles = ((M + BM - 1) / BM) * ((N + BN - 1) / BN);
    const size_t smem = Tile<BN>::total + 1024;
    static_assert(Tile<BN>::total + 1024 <= 227 * 1024, "the stages do not fit shared memory");
    static size_t attr[kMaxDevices] = {};
    CMLB_CUDA(cmlb_ensure_smem(gemm_bf16_kernel<BN>, smem, attr));
    CMLB_CUDA(launch_chain(gemm_bf16_kernel<BN>, dim3(tiles < cmlb_num_sms() ? tiles : cmlb_num_sms()), dim3(GEMM_THREADS), smem, 1, st, xmap, wmap, M,
                           N, W->cols, out, ex));
    return CMLB200_OK;
}

int gemm_entry(const cmlb200_dense* W, const uint16_t* x, int ldx, int x_rows, int M, int N, const GemmOut& out, const GemmExperts& ex, const char* who,
               void* stream) {
    CMLB_REQUIRE(W && W->w && x && out.y && M > 0, "%s: bad argument", who);
    CMLB_REQUIRE(W->dtype == CMLB200_DT_BF16 && W->rows > 0 && W->cols > 0 && W->ld % 8 == 0 && W->ld >= W->cols, "%s: bad weight [%d, %d], stride %d", who, W->rows, W->cols, W->ld);
    CMLB_REQUIRE(ldx % 8 == 0 && ldx >= W->cols && (((uintptr_t)x | (uintptr_t)W->w) & 15) == 0, "%s: x stride %d / alignment", who, ldx);
    // The widest tile moves the fewest bytes per flop; narrower ones spread a small product over more
    // SMs. Cost of a form: waves of tiles times its width, with the narrow forms' extra operand traffic.
    const int gm = (M + BM - 1) / BM, sms = cmlb_num_sms();
    auto waves = [&](int bn) { return (double)((gm * ((N + bn - 1) / bn) + sms - 1) / sms); };
    const double c256 = waves(256) * 256, c128 = waves(128) * 128 * 1.15, c64 = waves(64) * 64 * 1.6;
    cudaStream_t st = as_stream(stream);
    if (c256 <= c128 && c256 <= c64) return launch_gemm<256>(W, x, ldx, x_rows, M, N, out, ex, st);
    if (c128 <= c64) return launch_gemm<128>(W, x, ldx, x_rows, M, N, out, ex, st);
    return launch_gemm<64>(W, x, ldx, x_rows, M, N, out, ex, st);
}

// The plan's positions of `rows` step rows, and the most row tiles they can make.
int gemm_experts(const cmlb200_moe* m, const cmlb200_dense* W, const uint16_t* x, int ldx, int rows, GemmOut out, const char* who, void* stream) {
    CMLB_REQUIRE(m && m->experts > 0 && m->top > 0 && rows > 0 && W && W->rows % (16 * m->experts) == 0, "%s: bad argument", who);
    CMLB_REQUIRE(((uintptr_t)m->tiles & 15) == 0, "%s: the tile list must be 16-byte aligned", who);
    const long positions = cmlb200_moe_positions(rows, m->top, m->experts, BM);
    CMLB_REQUIRE(positions > 0 && positions < (1l << 30), "%s: %ld positions", who, positions);
    const GemmExperts ex = {(const int4*)m->tiles, m->num_tiles, W->rows / m->experts};
    return gemm_entry(W, x, ldx, (int)positions, (int)positions, ex.w_rows, out, ex, who, stream);
}

}  // namespace

extern "C" int cmlb200_gemm_dense(const cmlb200_dense* W, const uint16_t* d_x, int ldx, int M, float* d_y, int ldy, void* stream) {
    CMLB_REQUIRE(W && ldy >= W->rows, "cmlb200_gemm_dense: output stride %d", ldy);
    GemmOut out = {};
    out.form = OUT_F32; out.y = d_y; out.ldy = ldy; out.n_out = W->rows; out.bias = W->bias; out.cap = W->cap;
    return gemm_entry(W, d_x, ldx, M, M, W->rows, out, GemmExperts{}, "cmlb200_gemm_dense", stream);
}

extern "C" int cmlb200_gemm_dense_glu(const cmlb200_dense* W, const uint16_t* d_x, int ldx, int M, int ff, int act, uint16_t* d_f, int ldf, void* stream) {
    CMLB_REQUIRE(W && ff > 0 && W->rows == 2 * ((ff + 15) & ~15) && ldf >= ff, "cmlb200_gemm_dense_glu: weight rows do not fit %d outputs", ff);
    GemmOut out = {};
    out.form = OUT_GLU; out.act = act; out.y = d_f; out.ldy = ldf; out.n_out = ff;
    return gemm_entry(W, d_x, ldx, M, M, W->rows, out, GemmExperts{}, "cmlb200_gemm_dense_glu", stream);
}

extern "C" int cmlb200_moe_gemm(const cmlb200_moe* m, const cmlb200_dense* W, const uint16_t* d_x, int ldx, int rows, int n_out, float* d_y, int ldy,
                                void* stream) {
    CMLB_REQUIRE(m && W && n_out > 0 && n_out <= W->rows / m->experts && ldy >= n_out, "cmlb200_moe_gemm: %d outputs, stride %d", n_out, ldy);
    GemmOut out = {};
    out.form = OUT_F32; out.y = d_y; out.ldy = ldy; out.n_out = n_out;
    return gemm_experts(m, W, d_x, ldx, rows, out, "cmlb200_moe_gemm", stream);
}

extern "C" int cmlb200_moe_gemm_glu(const cmlb200_moe* m, const cmlb200_dense* W, const uint16_t* d_x, int ldx, int rows, int ff, int act, float limit,
                                    uint16_t* d_f, int ldf, void* stream) {
    CMLB_REQUIRE(m && W && ff > 0 && W->rows == m->experts * 2 * ((ff + 15) & ~15) && ldf >= ff, "cmlb200_moe_gemm_glu: weight rows do not fit %d outputs", ff);
    GemmOut out = {};
    out.form = OUT_GLU; out.act = act; out.limit = limit; out.y = d_f; out.ldy = ldf; out.n_out = ff;
    return gemm_experts(m, W, d_x, ldx, rows, out, "cmlb200_moe_gemm_glu", stream);
}

extern "C" int cmlb200_moe_gemm_act(const cmlb200_moe* m, const cmlb200_dense* W, const uint16_t* d_x, int ldx, int rows, int ff, int act, uint16_t* d_f, int ldf,
                                    void* stream) {
    CMLB_REQUIRE(m && W && ff > 0 && W->rows == m->experts * ((ff + 15) & ~15) && ldf >= ff, "cmlb200_moe_gemm_act: weight rows do not fit %d outputs", ff);
    CMLB_REQUIRE(act == CMLB200_ACT_SILU || act == CMLB200_ACT_GELU_TANH || act == CMLB200_ACT_GELU_ERF, "cmlb200_moe_gemm_act: activation %d", act);
    CMLB_REQUIRE(ldf % 2 == 0 && ((uintptr_t)d_f & 3) == 0, "cmlb200_moe_gemm_act: output stride %d", ldf);
    GemmOut out = {};
    out.form = OUT_ACT; out.act = act; out.y = d_f; out.ldy = ldf; out.n_out = ff;
    return gemm_experts(m, W, d_x, ldx, rows, out, "cmlb200_moe_gemm_act", stream);
}

extern "C" int cmlb200_latent_expand(const cmlb200_latent* a, const cmlb200_dense* W, const uint16_t* d_c_bf16, int rows, const cmlb200_attn* s, void* stream) {
    CMLB_REQUIRE(a && W && s && s->k_pool && s->cache_dtype == CMLB200_DT_F16, "cmlb200_latent_expand: bad argument");
    const int vp = (a->vdim + 15) & ~15;               // a head's value rows come padded, as cmlb200_latent_output reads them
    CMLB_REQUIRE(W->rows == a->heads * (a->dim + vp) && W->cols == a->rank && s->heads == a->heads && s->kv_heads == a->heads && s->dim == a->dim + a->rot_dim &&
                 s->vdim == a->vdim && s->dim_ld >= s->dim && s->vdim_ld >= vp, "cmlb200_latent_expand: shapes do not fit");
    GemmOut out = {};
    out.form = OUT_HEADS; out.y = s->v_pool; out.n_out = W->rows; out.keys = (__half*)s->k_pool;
    out.key_cols = a->heads * a->dim; out.dim = a->dim; out.dim_ld = s->dim_ld; out.ldk = a->heads * s->dim_ld;
    out.vdim = vp; out.vdim_ld = s->vdim_ld; out.ldy = a->heads * s->vdim_ld;
    return gemm_entry(W, d_c_bf16, a->ld_rank, rows, rows, W->rows, out, GemmExperts{}, "cmlb200_latent_expand", stream);
}

extern "C" int cmlb200_gemm_dense_status(int* status, int reset) {
    CMLB_REQUIRE(status, "cmlb200_gemm_dense_status: NULL argument");
    CMLB_CUDA(cudaDeviceSynchronize());
    CMLB_CUDA(cudaMemcpyFromSymbol(status, g_dense_status, sizeof(int)));
    if (reset) {
        const int zero = 0;
        CMLB_CUDA(cudaMemcpyToSymbol(g_dense_status, &zero, sizeof(int)));
    }
    return CMLB200_OK;
}
