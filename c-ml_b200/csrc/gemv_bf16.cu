// Decode product of dense bf16 weights, up to 32 rows of x: y[m][n] = sum_k x[m][k] W[n][k], bf16
// operands, fp32 sums. The weight streams from HBM once, straight into the A fragments of mma.sync
// m16n8k16: a thread's fragment needs pairs of neighbouring columns, and since any order of the columns
// will do as long as both operands use the same one, lane t of a quad takes columns 8t .. 8t + 7 and
// 32 + 8t .. 32 + 8t + 7 of every 64: two 16-byte loads per row feed four MMAs with no shared memory in
// between, and the quad reads 128 contiguous bytes per row. x fragments come the same way through L1.
// The eight warps of a CTA split K and meet in shared memory in a fixed order.
//
// The first weights are requested before the launch waits for its predecessor: they do not depend on it.
// W: [rows padded to 16][ldw], ldw a multiple of 64, zeros in the padding. x: [M][ldx], readable (and
// finite) up to column round_up(K, 64).
#include "lm_util.cuh"

namespace {

constexpr int GV_WARPS = 8;

// RT tiles of 16 weight rows per CTA, NB groups of 8 rows of x. GLU: tile 0 = 16 gate rows, tile 1 = the
// 16 up rows that go with them; the output is bf16 act(gate) * up.
// EXPERT: blockIdx.y counts the chosen experts; an expert's w_rows weight rows follow those of the one before it, its
// rows of x are those that chose it (m.src, or the positions themselves), and y has a row per position. Without a gate its
// output is fp32, or bf16 act(y) where act is not negative.
struct GemvExperts {
    cmlb200_moe m;
    int w_rows, gather;
};
template <int RT, int NB, bool GLU, bool EXPERT>
__global__ void __launch_bounds__(GV_WARPS * 32)
gemv_bf16_kernel(const __nv_bfloat16* __restrict__ W, int ldw, const __nv_bfloat16* __restrict__ x, int ldx, int M, int N, int K, int act,
                 float limit, const float* __restrict__ bias, float cap, void* __restrict__ y, int ldy, const GemvExperts ex) {
    __shared__ float part[GV_WARPS][RT * 16][NB * 8 + 1];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
    const int n0 = blockIdx.x * RT * 16;
    const int chunks = (K + 63) / 64;
    int first = 0;
    if (EXPERT) {                                       // which weights are needed is known only now
        dep_wait();
        dep_trigger();
        if ((int)blockIdx.y >= *ex.m.num_active) return;
        const int e = ex.m.active[blockIdx.y];
        first = ex.m.start[e];
        M = ex.m.count[e];
        W += (size_t)e * ex.w_rows * ldw;
    }
    const __nv_bfloat16* wrow[RT][2];
#pragma unroll
    for (int i = 0; i < RT; i++) {
        wrow[i][0] = W + (size_t)(n0 + i * 16 + g) * ldw + 8 * t;
        wrow[i][1] = wrow[i][0] + (size_t)8 * ldw;
    }
    constexpr int RING = 4 / RT;                        // 64-column chunks in flight per warp
    uint4 w[RING][RT][2][2];
    auto fetch = [&](int u, int c) {
#pragma unroll
        for (int i = 0; i < RT; i++)
#pragma unroll
            for (int e = 0; e < 2; e++)
#pragma unroll
                for (int s = 0; s < 2; s++)
                    w[u][i][e][s] = c < chunks ? ld_stream(wrow[i][e] + (size_t)c * 64 + 32 * s) : make_uint4(0u, 0u, 0u, 0u);
    };
#pragma unroll
    for (int u = 0; u < RING; u++) fetch(u, warp + u * GV_WARPS);
    if (!EXPERT) {
        dep_wait();
        dep_trigger();
    }
    float acc[RT][NB][4];
#pragma unroll
    for (int i = 0; i < RT; i++)
#pragma unroll
        for (int b = 0; b < NB; b++) { acc[i][b][0] = 0.f; acc[i][b][1] = 0.f; acc[i][b][2] = 0.f; acc[i][b][3] = 0.f; }
    const __nv_bfloat16* xr[NB];
#pragma unroll
    for (int b = 0; b < NB; b++) {                      // rows past M repeat the last, never stored
        int r = min(b * 8 + g, M - 1);
        if (EXPERT) r = ex.gather ? ex.m.src[first + r] : first + r;
        xr[b] = x + (size_t)r * ldx + 8 * t;
    }
    for (int c0 = warp; c0 < chunks; c0 += RING * GV_WARPS) {
#pragma unroll
        for (int u = 0; u < RING; u++) {
            const int c = min(c0 + u * GV_WARPS, chunks - 1);         // past the end: zero weights
#pragma unroll
            for (int b = 0; b < NB; b++) {
                if (EXPERT && b * 8 >= M) continue;
                const uint4 x0 = *reinterpret_cast<const uint4*>(xr[b] + (size_t)c * 64), x1 = *reinterpret_cast<const uint4*>(xr[b] + (size_t)c * 64 + 32);
#pragma unroll
                for (int i = 0; i < RT; i++) {
                    mma_bf16(acc[i][b], w[u][i][0][0].x, w[u][i][1][0].x, w[u][i][0][0].y, w[u][i][1][0].y, x0.x, x0.y);
                    mma_bf16(acc[i][b], w[u][i][0][0].z, w[u][i][1][0].z, w[u][i][0][0].w, w[u][i][1][0].w, x0.z, x0.w);
                    mma_bf16(acc[i][b], w[u][i][0][1].x, w[u][i][1][1].x, w[u][i][0][1].y, w[u][i][1][1].y, x1.x, x1.y);
                    mma_bf16(acc[i][b], w[u][i][0][1].z, w[u][i][1][1].z, w[u][i][0][1].w, w[u][i][1][1].w, x1.z, x1.w);
                }
            }
            fetch(u, c0 + (u + RING) * GV_WARPS);
        }
    }
    // accumulator register 0, 1: weight row g, rows 2t, 2t + 1 of x; 2, 3: weight row g + 8
#pragma unroll
    for (int i = 0; i < RT; i++)
#pragma unroll
        for (int b = 0; b < NB; b++) {
            part[warp][i * 16 + g][b * 8 + 2 * t] = acc[i][b][0];
            part[warp][i * 16 + g][b * 8 + 2 * t + 1] = acc[i][b][1];
            part[warp][i * 16 + g + 8][b * 8 + 2 * t] = acc[i][b][2];
            part[warp][i * 16 + g + 8][b * 8 + 2 * t + 1] = acc[i][b][3];
        }
    __syncthreads();
    constexpr int OUT = GLU ? 16 : RT * 16;
    for (int i = threadIdx.x; i < OUT * NB * 8; i += GV_WARPS * 32) {
        const int n = i % OUT, m = i / OUT;
        if (m >= M) break;
        float s = 0.f, s2 = 0.f;
#pragma unroll
        for (int k = 0; k < GV_WARPS; k++) {
            s += part[k][n][m];
            if (GLU) s2 += part[k][RT * 16 - 16 + n][m];
        }
        if (GLU) {
            const int c = blockIdx.x * 16 + n;
            if (c < N) static_cast<__nv_bfloat16*>(y)[(size_t)(first + m) * ldy + c] = __float2bfloat16_rn(glu_act_fast(act, s, s2, limit));
        } else if (n0 + n < N) {
            if (!EXPERT && bias) s += bias[n0 + n];
            if (!EXPERT && cap > 0.f) s = soft_cap(s, cap);
            if (EXPERT && act >= 0) static_cast<__nv_bfloat16*>(y)[(size_t)(first + m) * ldy + n0 + n] = __float2bfloat16_rn(unary_act_fast(act, s));
            else static_cast<float*>(y)[(size_t)(first + m) * ldy + n0 + n] = s;
        }
    }
}

template <int RT, bool GLU>
int launch_gemv(const cmlb200_dense* W, const uint16_t* x, int ldx, int M, int act, void* y, int ldy, int n_out, cudaStream_t st) {
    const dim3 grid((unsigned)((W->rows + RT * 16 - 1) / (RT * 16)));
    const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(W->w);
    const __nv_bfloat16* xb = reinterpret_cast<const __nv_bfloat16*>(x);
#define GV_LAUNCH(NB) CMLB_CUDA(launch_chain(gemv_bf16_kernel<RT, NB, GLU, false>, grid, dim3(GV_WARPS * 32), 0, 1, st, w, W->ld, xb, ldx, M, n_out, W->cols, act, 0.f, W->bias, W->cap, y, ldy, GemvExperts{}))
    if (M <= 8) GV_LAUNCH(1);
    else if (M <= 16) GV_LAUNCH(2);
    else GV_LAUNCH(4);
#undef GV_LAUNCH
    return CMLB200_OK;
}

template <int RT, bool GLU>
int launch_gemv_experts(const cmlb200_moe* m, const cmlb200_dense* W, const uint16_t* x, int ldx, int gather, int rows, int act, float limit, void* y,
                        int ldy, int n_out, cudaStream_t st) {
    const int per = W->rows / m->experts, pairs = rows * m->top;
    const dim3 grid((unsigned)((GLU ? (per + 31) / 32 : (n_out + 15) / 16)), (unsigned)(pairs < m->experts ? pairs : m->experts));
    const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(W->w);
    const __nv_bfloat16* xb = reinterpret_cast<const __nv_bfloat16*>(x);
    const GemvExperts ex = {*m, per, gather};
#define GE_LAUNCH(NB) CMLB_CUDA(launch_chain(gemv_bf16_kernel<RT, NB, GLU, true>, grid, dim3(GV_WARPS * 32), 0, 1, st, w, W->ld, xb, ldx, rows, n_out, W->cols, act, limit, (const float*)nullptr, 0.f, y, ldy, ex))
    if (rows <= 8) GE_LAUNCH(1);
    else if (rows <= 16) GE_LAUNCH(2);
    else GE_LAUNCH(4);
#undef GE_LAUNCH
    return CMLB200_OK;
}

int check_gemv(const cmlb200_dense* W, const uint16_t* x, int ldx, int M, void* y, const char* who) {
    CMLB_REQUIRE(W && W->w && x && y, "%s: NULL argument", who);
    CMLB_REQUIRE(W->dtype == CMLB200_DT_BF16 && W->rows > 0 && W->cols > 0 && W->ld % 64 == 0 && W->ld >= W->cols, "%s: bad weight [%d, %d], stride %d", who, W->rows, W->cols, W->ld);
    CMLB_REQUIRE(M >= 1 && M <= 32, "%s: M=%d outside 1..32", who, M);
    CMLB_REQUIRE(ldx % 8 == 0 && ldx >= W->ld && (((uintptr_t)x | (uintptr_t)W->w) & 15) == 0, "%s: x needs a stride of at least %d and 16-byte alignment", who, W->ld);
    return CMLB200_OK;
}

}  // namespace

extern "C" int cmlb200_gemv_dense(const cmlb200_dense* W, const uint16_t* d_x, int ldx, int M, float* d_y, int ldy, void* stream) {
    const int rc = check_gemv(W, d_x, ldx, M, d_y, "cmlb200_gemv_dense");
    if (rc) return rc;
    CMLB_REQUIRE(ldy >= W->rows, "cmlb200_gemv_dense: output stride %d", ldy);
    return launch_gemv<1, false>(W, d_x, ldx, M, 0, d_y, ldy, W->rows, as_stream(stream));
}

extern "C" int cmlb200_gemv_dense_glu(const cmlb200_dense* W, const uint16_t* d_x, int ldx, int M, int ff, int act, uint16_t* d_f, int ldf, void* stream) {
    const int rc = check_gemv(W, d_x, ldx, M, d_f, "cmlb200_gemv_dense_glu");
    if (rc) return rc;
    CMLB_REQUIRE(ff > 0 && W->rows == 2 * ((ff + 15) & ~15) && ldf >= ff, "cmlb200_gemv_dense_glu: %d weight rows for %d outputs", W->rows, ff);
    return launch_gemv<2, true>(W, d_x, ldx, M, act, d_f, ldf, ff, as_stream(stream));
}

extern "C" int cmlb200_moe_gemv(const cmlb200_moe* m, const cmlb200_dense* W, const uint16_t* d_x, int ldx, int gather, int rows, int n_out, float* d_y,
                                int ldy, void* stream) {
    const int rc = check_gemv(W, d_x, ldx, rows, d_y, "cmlb200_moe_gemv");
    if (rc) return rc;
    CMLB_REQUIRE(m && m->experts > 0 && m->experts <= 65535 && W->rows % (16 * m->experts) == 0 && n_out > 0 && n_out <= W->rows / m->experts && ldy >= n_out,
                 "cmlb200_moe_gemv: %d weight rows, %d outputs, stride %d", W->rows, n_out, ldy);
    return launch_gemv_experts<1, false>(m, W, d_x, ldx, gather, rows, -1, 0.f, d_y, ldy, n_out, as_stream(stream));
}

extern "C" int cmlb200_moe_gemv_glu(const cmlb200_moe* m, const cmlb200_dense* W, const uint16_t* d_x, int ldx, int gather, int rows, int ff, int act,
                                    float limit, uint16_t* d_f, int ldf, void* stream) {
    const int rc = check_gemv(W, d_x, ldx, rows, d_f, "cmlb200_moe_gemv_glu");
    if (rc) return rc;
    CMLB_REQUIRE(m && m->experts > 0 && m->experts <= 65535 && ff > 0 && W->rows == m->experts * 2 * ((ff + 15) & ~15) && ldf >= ff,
                 "cmlb200_moe_gemv_glu: %d weight rows for %d outputs", W->rows, ff);
    return launch_gemv_experts<2, true>(m, W, d_x, ldx, gather, rows, act, limit, d_f, ldf, ff, as_stream(stream));
}

extern "C" int cmlb200_moe_gemv_act(const cmlb200_moe* m, const cmlb200_dense* W, const uint16_t* d_x, int ldx, int gather, int rows, int ff, int act, uint16_t* d_f,
                                    int ldf, void* stream) {
    const int rc = check_gemv(W, d_x, ldx, rows, d_f, "cmlb200_moe_gemv_act");
    if (rc) return rc;
    CMLB_REQUIRE(m && m->experts > 0 && m->experts <= 65535 && ff > 0 && W->rows == m->experts * ((ff + 15) & ~15) && ldf >= ff,
                 "cmlb200_moe_gemv_act: %d weight rows for %d outputs", W->rows, ff);
    CMLB_REQUIRE(act == CMLB200_ACT_SILU || act == CMLB200_ACT_GELU_TANH || act == CMLB200_ACT_GELU_ERF, "cmlb200_moe_gemv_act: activation %d", act);
    return launch_gemv_experts<1, false>(m, W, d_x, ldx, gather, rows, act, 0.f, d_f, ldf, ff, as_stream(stream));
}
