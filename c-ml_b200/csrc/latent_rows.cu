// Row-wise pieces of latent attention (cmlb200_latent): the cache append (norm of the latent, rotation of the shared
// key part) with the rotation of the queries; the two per-head products around attention over latents
// (q -> Wuk^T q in front, o -> Wuv o with the gate, per element or per head, behind); and the gathering of a long portion's latents
// for the expansion into per-head keys and values. Norms, angles and rotations are fp32.
#include "lm_util.cuh"

namespace {

// Where the rotated queries of a row go: base + head * head_ld + off + i, times mul; entries up to off + fill are zeroed.
template <typename TQ>
struct QueryOut {
    TQ* base;
    int head_ld, off, fill;
    float mul;
};

__device__ __forceinline__ void store2(float* d, float x, float y) { *reinterpret_cast<float2*>(d) = make_float2(x, y); }
__device__ __forceinline__ void store2(__half* d, float x, float y) {
    const __half v[2] = {narrow<__half>(x), narrow<__half>(y)};
    *reinterpret_cast<uint32_t*>(d) = *reinterpret_cast<const uint32_t*>(v);
}

// A block's work on one projection row, or part `part` of it (the first one fills the cache). cs: rot_dim floats, red: 32.
template <typename KV, typename TQ>
__device__ __forceinline__ void latent_row(const cmlb200_latent& a, const float* row, int p, int slot, const QueryOut<TQ>& q, int part, int parts, float* cs,
                                           float* red) {
    const bool fill = a.kv_col >= 0 && part == 0;
    const int half = a.rot_dim / 2, nt = blockDim.x;
    for (int i = threadIdx.x; i < half; i += nt) {
        float s, c;
        sincosf((float)p * a.freq[i], &s, &c);
        cs[i] = c * a.rot_mul;
        cs[half + i] = s * a.rot_mul;
    }
    float inv = 0.f;
    const float* kv = row + a.kv_col;
    if (fill) {
        const float ss = block_sum(square_share(kv, a.rank), red);
        inv = 1.0f / sqrtf(ss / (float)a.rank + a.eps);
    } else {
        __syncthreads();
    }
    __syncthreads();
    if (fill) {
        const size_t at = (size_t)a.block_table[(size_t)slot * a.table_ld + p / a.block_size] * a.block_size + p % a.block_size;
        KV* d = static_cast<KV*>(a.pool) + at * a.ld;
#pragma unroll 4
        for (int i = threadIdx.x; i < a.rank; i += nt) d[i] = narrow<KV>(kv[i] * inv * a.c_norm[i]);
        for (int i = threadIdx.x; i < half; i += nt) {
            const float u = kv[a.rank + i], v = kv[a.rank + half + i];
            d[a.rank + i] = narrow<KV>(u * cs[i] - v * cs[half + i]);
            d[a.rank + half + i] = narrow<KV>(v * cs[i] + u * cs[half + i]);
        }
        for (int i = a.rank + a.rot_dim + threadIdx.x; i < a.ld; i += nt) d[i] = narrow<KV>(0.f);
    }
    const int hd = a.dim + a.rot_dim, first = part * nt + threadIdx.x, step = parts * nt;
    // two neighbouring pairs at a time where everything is aligned for it
    if ((half & 1) == 0 && ((a.dim | hd | q.head_ld | q.off) & 1) == 0 && (((uintptr_t)row | ((uintptr_t)q.base * (8 / (2 * sizeof(TQ))))) & 7) == 0) {
        const int h2 = half >> 1;
#pragma unroll 4
        for (int j = first; j < a.heads * h2; j += step) {
            const int h = j / h2, i = (j - h * h2) * 2;
            const float* s = row + h * hd + a.dim;
            const float2 u = *reinterpret_cast<const float2*>(s + i), v = *reinterpret_cast<const float2*>(s + half + i);
            const float2 c = *reinterpret_cast<const float2*>(cs + i), n = *reinterpret_cast<const float2*>(cs + half + i);
            TQ* d = q.base + (size_t)h * q.head_ld + q.off;
            store2(d + i, (u.x * c.x - v.x * n.x) * q.mul, (u.y * c.y - v.y * n.y) * q.mul);
            store2(d + half + i, (v.x * c.x + u.x * n.x) * q.mul, (v.y * c.y + u.y * n.y) * q.mul);
        }
    } else {
        for (int j = first; j < a.heads * half; j += step) {
            const int h = j / half, i = j - h * half;
            const float* s = row + h * hd + a.dim;
            const float u = s[i], v = s[half + i];
            TQ* d = q.base + (size_t)h * q.head_ld + q.off;
            d[i] = narrow<TQ>((u * cs[i] - v * cs[half + i]) * q.mul);
            d[half + i] = narrow<TQ>((v * cs[i] + u * cs[half + i]) * q.mul);
        }
    }
    const int pad = q.fill - a.rot_dim;
    for (int j = first; j < a.heads * pad; j += step) {
        const int h = j / pad;
        q.base[(size_t)h * q.head_ld + q.off + a.rot_dim + j - h * pad] = narrow<TQ>(0.f);
    }
}

// grid = rows. TQ float: the queries turn in place (mul 1) or go to rows of their own (q_out, stride q_ld).
template <typename KV>
__global__ void __launch_bounds__(256)
latent_append_kernel(const cmlb200_latent a, float* proj, int ld, const int* __restrict__ row_pos, const int* __restrict__ row_slot, float* q_out,
                     size_t q_ld, int head_ld, int off) {
    extern __shared__ float cs[];
    __shared__ float red[32];
    dep_wait();
    dep_trigger();
    const int r = blockIdx.x;
    float* row = proj + (size_t)r * ld;
    const QueryOut<float> q = {q_out ? q_out + (size_t)r * q_ld : row, head_ld, off, a.rot_dim, 1.0f};
    latent_row<KV, float>(a, row, row_pos[r], row_slot[r], q, 0, 1, cs, red);
}

constexpr int LQ_WARPS = 4, LQ_THREADS = LQ_WARPS * 32, LQ_COLS = LQ_WARPS * 16, LQ_ROWS = 32;

__host__ __device__ inline int row_parts(int rows) { return rows <= 8 ? 4 : 1; }      // blocks that share a row's rotation

// grid = (rank / 64, heads + extra, rows / 32). Blocks y < heads: q16[row][y][n] = scale log2 e sum_d q[row][y][d] Wuk[y][d][n],
// a warp per 16 outputs n, up to 32 rows. The blocks behind them: latent_row of the same rows.
template <int NB>
__global__ void __launch_bounds__(LQ_THREADS)
latent_query_kernel(const cmlb200_latent a, const __nv_bfloat16* __restrict__ wukt, const float* __restrict__ proj, int ld, const int* __restrict__ row_pos,
                    const int* __restrict__ row_slot, int rows, __half* __restrict__ q16) {
    extern __shared__ __align__(16) uint8_t sm[];
    __shared__ float red[32];
    const int r0 = blockIdx.z * LQ_ROWS, n = min(LQ_ROWS, rows - r0), hd = a.dim + a.rot_dim;
    const float mul = a.scale * kLog2e;
    if ((int)blockIdx.y >= a.heads) {
        dep_wait();
        dep_trigger();
        const int job = (blockIdx.y - a.heads) * gridDim.x + blockIdx.x, parts = row_parts(rows), r = r0 + job / parts;
        if (r >= r0 + n) return;
        const QueryOut<__half> q = {q16 + (size_t)r * a.heads * a.ld, a.ld, a.rank, a.ld - a.rank, mul};
        latent_row<__half, __half>(a, proj + (size_t)r * ld, row_pos[r], row_slot[r], q, job % parts, parts, reinterpret_cast<float*>(sm), red);
        return;
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3, h = blockIdx.y;
    const int dp = (a.dim + 63) & ~63, rp = (a.rank + 15) & ~15, lx = dp + 8;
    __nv_bfloat16* xs = reinterpret_cast<__nv_bfloat16*>(sm);           // [NB * 8][lx]
    __half* os = reinterpret_cast<__half*>(xs + NB * 8 * lx);           // [NB * 8][LQ_COLS + 8]
    const int n0 = blockIdx.x * LQ_COLS + warp * 16;
    const bool live = n0 < rp;
    const __nv_bfloat16* w0 = wukt + ((size_t)h * rp + (live ? n0 : 0) + g) * dp + 8 * t;
    const __nv_bfloat16* w1 = w0 + (size_t)8 * dp;
    uint4 w[2][2][2];                                   // two 64-column chunks in flight
    auto fetch = [&](int u, int c) {
#pragma unroll
        for (int s = 0; s < 2; s++) {
            w[u][0][s] = c < dp ? ld_stream(w0 + c + 32 * s) : make_uint4(0u, 0u, 0u, 0u);
            w[u][1][s] = c < dp ? ld_stream(w1 + c + 32 * s) : make_uint4(0u, 0u, 0u, 0u);
        }
    };
    fetch(0, 0);
    fetch(1, 64);
    dep_wait();
    dep_trigger();
    for (int d = threadIdx.x; d < dp; d += LQ_THREADS) {
#pragma unroll
        for (int m = 0; m < NB * 8; m++) xs[m * lx + d] = __float2bfloat16_rn(m < n && d < a.dim ? proj[(size_t)(r0 + m) * ld + h * hd + d] : 0.f);
    }
    __syncthreads();
    float acc[NB][4];
#pragma unroll
    for (int b = 0; b < NB; b++) { acc[b][0] = 0.f; acc[b][1] = 0.f; acc[b][2] = 0.f; acc[b][3] = 0.f; }
    for (int c0 = 0; c0 < dp; c0 += 128) {
#pragma unroll
        for (int u = 0; u < 2; u++) {
            const int c = min(c0 + u * 64, dp - 64);    // past the end: zero weights
#pragma unroll
            for (int b = 0; b < NB; b++) {
                const __nv_bfloat16* x = xs + (b * 8 + g) * lx + c + 8 * t;
                const uint4 x0 = *reinterpret_cast<const uint4*>(x), x1 = *reinterpret_cast<const uint4*>(x + 32);
                mma_bf16(acc[b], w[u][0][0].x, w[u][1][0].x, w[u][0][0].y, w[u][1][0].y, x0.x, x0.y);
                mma_bf16(acc[b], w[u][0][0].z, w[u][1][0].z, w[u][0][0].w, w[u][1][0].w, x0.z, x0.w);
                mma_bf16(acc[b], w[u][0][1].x, w[u][1][1].x, w[u][0][1].y, w[u][1][1].y, x1.x, x1.y);
                mma_bf16(acc[b], w[u][0][1].z, w[u][1][1].z, w[u][0][1].w, w[u][1][1].w, x1.z, x1.w);
            }
            fetch(u, c0 + 128 + u * 64);
        }
    }
    constexpr int LO = LQ_COLS + 8;
#pragma unroll
    for (int b = 0; b < NB; b++)
#pragma unroll
        for (int e = 0; e < 4; e++) os[(b * 8 + 2 * t + (e & 1)) * LO + warp * 16 + g + (e >> 1) * 8] = narrow<__half>(acc[b][e] * mul);
    __syncthreads();
    for (int i = threadIdx.x; i < n * LQ_COLS; i += LQ_THREADS) {
        const int m = i / LQ_COLS, c = i - m * LQ_COLS, col = blockIdx.x * LQ_COLS + c;
        if (col < a.rank) q16[((size_t)(r0 + m) * a.heads + h) * a.ld + col] = os[m * LO + c];
    }
}

constexpr int LO_WARPS = 8;

// grid = (vdim / 16, heads, rows / 32): out[row][h * vdim + v] = sum_r o[row][h][r] Wuv[h][v][r] (times the gate's
// sigmoid). The eight warps split the latent and meet in shared memory in a fixed order.
template <int NB>
__global__ void __launch_bounds__(LO_WARPS * 32)
latent_output_kernel(const cmlb200_latent a, const __nv_bfloat16* __restrict__ wuv, const __nv_bfloat16* __restrict__ o, const float* __restrict__ proj,
                     int ld, int rows, __nv_bfloat16* __restrict__ out, int out_ld) {
    __shared__ float part[LO_WARPS][16][NB * 8 + 1];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3, h = blockIdx.y, n0 = blockIdx.x * 16;
    const int r0 = blockIdx.z * LQ_ROWS, n = min(LQ_ROWS, rows - r0), vp = (a.vdim + 15) & ~15, chunks = a.ld_rank / 64;
    const __nv_bfloat16* w0 = wuv + ((size_t)h * vp + n0 + g) * a.ld_rank + 8 * t;
    const __nv_bfloat16* w1 = w0 + (size_t)8 * a.ld_rank;
    uint4 w[2][2];
    auto fetch = [&](int c) {
#pragma unroll
        for (int s = 0; s < 2; s++) {
            w[0][s] = c < chunks ? ld_stream(w0 + (size_t)c * 64 + 32 * s) : make_uint4(0u, 0u, 0u, 0u);
            w[1][s] = c < chunks ? ld_stream(w1 + (size_t)c * 64 + 32 * s) : make_uint4(0u, 0u, 0u, 0u);
        }
    };
    fetch(warp);
    dep_wait();
    dep_trigger();
    float acc[NB][4];
    const __nv_bfloat16* xr[NB];
#pragma unroll
    for (int b = 0; b < NB; b++) {
        acc[b][0] = 0.f; acc[b][1] = 0.f; acc[b][2] = 0.f; acc[b][3] = 0.f;
        xr[b] = o + ((size_t)(r0 + min(b * 8 + g, n - 1)) * a.heads + h) * a.ld_rank + 8 * t;
    }
    for (int c = warp; c < chunks; c += LO_WARPS) {
#pragma unroll
        for (int b = 0; b < NB; b++) {
            const uint4 x0 = *reinterpret_cast<const uint4*>(xr[b] + (size_t)c * 64), x1 = *reinterpret_cast<const uint4*>(xr[b] + (size_t)c * 64 + 32);
            mma_bf16(acc[b], w[0][0].x, w[1][0].x, w[0][0].y, w[1][0].y, x0.x, x0.y);
            mma_bf16(acc[b], w[0][0].z, w[1][0].z, w[0][0].w, w[1][0].w, x0.z, x0.w);
            mma_bf16(acc[b], w[0][1].x, w[1][1].x, w[0][1].y, w[1][1].y, x1.x, x1.y);
            mma_bf16(acc[b], w[0][1].z, w[1][1].z, w[0][1].w, w[1][1].w, x1.z, x1.w);
        }
        fetch(c + LO_WARPS);
    }
#pragma unroll
    for (int b = 0; b < NB; b++)
#pragma unroll
        for (int e = 0; e < 4; e++) part[warp][g + (e >> 1) * 8][b * 8 + 2 * t + (e & 1)] = acc[b][e];
    __syncthreads();
    for (int i = threadIdx.x; i < 16 * n; i += LO_WARPS * 32) {
        const int v = i % 16, m = i / 16, col = h * a.vdim + n0 + v;
        if (n0 + v >= a.vdim) continue;
        float s = 0.f;
#pragma unroll
        for (int k = 0; k < LO_WARPS; k++) s += part[k][v][m];
        if (a.gate_col >= 0) s *= sigmoidf(proj[(size_t)(r0 + m) * ld + a.gate_col + (a.gate_heads ? h : col)]);
        out[(size_t)(r0 + m) * out_ld + col] = __float2bfloat16_rn(s);
    }
}

// 32-bit per-head product, a warp per output: y[r][h * y_ld + n] = sum_k x[r][h * x_ld + k] W[h][n][k], times the
// sigmoid of gate[r][h * N + n], or of gate[r][h]. grid = (N / 8, heads, rows).
__global__ void __launch_bounds__(256)
heads_linear_f32_kernel(const float* __restrict__ W, int N, int K, const float* __restrict__ x, size_t x_row, int x_ld, const float* __restrict__ gate,
                        size_t gate_row, int gate_heads, float* __restrict__ y, size_t y_row, int y_ld) {
    dep_wait();
    dep_trigger();
    const int n = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, h = blockIdx.y;
    if (n >= N) return;
    const float* w = W + ((size_t)h * N + n) * K;
    const float* xr = x + blockIdx.z * x_row + (size_t)h * x_ld;
    float s = 0.f;
    for (int k = lane; k < K; k += 32) s = fmaf(w[k], xr[k], s);
    s = lane_sum(s);
    if (gate) s *= sigmoidf(gate[blockIdx.z * gate_row + (gate_heads ? (size_t)h : (size_t)h * N + n)]);
    if (lane == 0) y[blockIdx.z * y_row + (size_t)h * y_ld + n] = s;
}

struct GatherList {
    int4 k[16];                                         // {slot, first key, keys, first scratch row}
};

// grid = (blocks of keys, sequences, parts): the latent as bf16 (zeros up to ld_rank), the shared key part into every
// head's key row behind its `dim` columns (heads shared out over the parts), and the block's entry of the scratch's block
// table. VEC: 8 elements at a time.
template <bool VEC>
__global__ void __launch_bounds__(256)
latent_gather_kernel(const cmlb200_latent a, const GatherList list, __nv_bfloat16* __restrict__ c, __half* __restrict__ keys, int dim_ld,
                     int* __restrict__ table, int table_ld) {
    dep_wait();
    dep_trigger();
    const int4 it = list.k[blockIdx.y];
    const int bs = a.block_size, b = blockIdx.x;
    if (b * bs >= it.z) return;
    const int blk = it.y / bs + b;
    if (threadIdx.x == 0) table[(size_t)it.x * table_ld + blk] = it.w / bs + b;
    const size_t from = (size_t)a.block_table[(size_t)it.x * a.table_ld + blk] * bs;
    const int n = min(bs, it.z - b * bs), tail = dim_ld - a.dim, h0 = blockIdx.z, hs = gridDim.z;
    const size_t row0 = (size_t)it.w + b * bs;
    const __half* pool = static_cast<const __half*>(a.pool) + from * a.ld;
    if (VEC) {
        const int c8 = a.ld_rank >> 3, t8 = tail >> 3;
        for (int j = blockIdx.z * 256 + threadIdx.x; j < n * c8; j += 256 * hs) {
            const int i = j / c8, d = (j - i * c8) * 8;
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (d < a.rank) {
                const uint4 w = *reinterpret_cast<const uint4*>(pool + (size_t)i * a.ld + d);
                const __half2* x = reinterpret_cast<const __half2*>(&w);
                __nv_bfloat162* y = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
                for (int e = 0; e < 4; e++) { const float2 f = __half22float2(x[e]); y[e] = __floats2bfloat162_rn(f.x, f.y); }
            }
            *reinterpret_cast<uint4*>(c + (row0 + i) * a.ld_rank + d) = v;
        }
        for (int j = threadIdx.x; j < n * t8; j += 256) {
            const int i = j / t8, d = (j - i * t8) * 8;
            const uint4 v = d < a.rot_dim ? *reinterpret_cast<const uint4*>(pool + (size_t)i * a.ld + a.rank + d) : make_uint4(0u, 0u, 0u, 0u);
            __half* k = keys + (row0 + i) * a.heads * dim_ld + a.dim + d;
            for (int h = h0; h < a.heads; h += hs) *reinterpret_cast<uint4*>(k + (size_t)h * dim_ld) = v;
        }
        return;
    }
    for (int j = blockIdx.z * 256 + threadIdx.x; j < n * a.ld_rank; j += 256 * hs) {
        const int i = j / a.ld_rank, d = j - i * a.ld_rank;
        c[(row0 + i) * a.ld_rank + d] = __float2bfloat16_rn(d < a.rank ? __half2float(pool[(size_t)i * a.ld + d]) : 0.f);
    }
    for (int j = threadIdx.x; j < n * tail; j += 256) {
        const int i = j / tail, d = j - i * tail;
        const __half v = d < a.rot_dim ? pool[(size_t)i * a.ld + a.rank + d] : __float2half_rn(0.f);
        __half* k = keys + (row0 + i) * a.heads * dim_ld + a.dim + d;
        for (int h = h0; h < a.heads; h += hs) k[(size_t)h * dim_ld] = v;
    }
}

int check_latent(const cmlb200_latent* a, int ld, const char* who) {
    CMLB_REQUIRE(a && a->heads > 0 && a->heads < 65535 && a->dim > 0 && a->rot_dim > 0 && a->rot_dim % 2 == 0 && a->vdim > 0 && a->rank > 0, "%s: bad sizes", who);
    CMLB_REQUIRE(a->ld >= a->rank + a->rot_dim && a->ld % 16 == 0 && a->ld_rank >= a->rank && a->ld_rank % 64 == 0, "%s: strides %d / %d", who, a->ld, a->ld_rank);
    CMLB_REQUIRE(a->freq && a->pool && a->block_table && a->table_ld > 0 && ((uintptr_t)a->pool & 15) == 0, "%s: no cache or frequencies", who);
    CMLB_REQUIRE(a->block_size >= 16 && (a->block_size & (a->block_size - 1)) == 0, "%s: block size %d must be a power of two >= 16", who, a->block_size);
    CMLB_REQUIRE(a->kv_col < 0 || a->c_norm, "%s: no norm weights", who);
    CMLB_REQUIRE(ld >= a->heads * (a->dim + a->rot_dim) && (a->kv_col < 0 || ld >= a->kv_col + a->rank + a->rot_dim) &&
                 (a->gate_col < 0 || ld >= a->gate_col + a->heads * (a->gate_heads ? 1 : a->vdim)), "%s: row stride %d", who, ld);
    CMLB_REQUIRE(a->rot_dim <= 8192, "%s: rotated size %d", who, a->rot_dim);
    return CMLB200_OK;
}

}  // namespace

extern "C" int cmlb200_latent_append(const cmlb200_latent* a, float* d_proj, int ld, const int* d_row_pos, const int* d_row_slot, int rows, void* stream) {
    const int rc = check_latent(a, ld, "cmlb200_latent_append");
    if (rc) return rc;
    CMLB_REQUIRE(d_proj && d_row_pos && d_row_slot && rows > 0, "cmlb200_latent_append: bad argument");
    const size_t smem = (size_t)a->rot_dim * 4;
    cudaStream_t st = as_stream(stream);
#define LA_LAUNCH(KV) CMLB_CUDA(launch_chain(latent_append_kernel<KV>, dim3(rows), dim3(256), smem, 1, st, *a, d_proj, ld, d_row_pos, d_row_slot, (float*)nullptr, (size_t)0, a->dim + a->rot_dim, a->dim))
    if (a->cache_dtype == CMLB200_DT_F32) LA_LAUNCH(float);
    else LA_LAUNCH(__half);
#undef LA_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_latent_query(const cmlb200_latent* a, const uint16_t* d_wukt, const float* d_proj, int ld, const int* d_row_pos, const int* d_row_slot,
                                    int rows, uint16_t* d_q_f16, void* stream) {
    const int rc = check_latent(a, ld, "cmlb200_latent_query");
    if (rc) return rc;
    CMLB_REQUIRE(d_wukt && d_proj && d_row_pos && d_row_slot && rows > 0 && d_q_f16 && a->cache_dtype == CMLB200_DT_F16, "cmlb200_latent_query: bad argument");
    CMLB_REQUIRE(((uintptr_t)d_wukt & 15) == 0 && rows <= 65535 * LQ_ROWS, "cmlb200_latent_query: alignment or %d rows", rows);
    const int gx = (a->rank + LQ_COLS - 1) / LQ_COLS, most = rows < LQ_ROWS ? rows : LQ_ROWS;
    const int jobs = most * row_parts(rows);
    const dim3 grid(gx, a->heads + (jobs + gx - 1) / gx, (rows + LQ_ROWS - 1) / LQ_ROWS);
    const int nb = rows <= 8 ? 1 : (rows <= 16 ? 2 : 4);
    const size_t x = (size_t)nb * 8 * (((a->dim + 63) & ~63) + 8) * 2 + (size_t)nb * 8 * (LQ_COLS + 8) * 2, rot = (size_t)a->rot_dim * 4;
    const size_t smem = x > rot ? x : rot;
    static size_t attr[3][kMaxDevices] = {};
    cudaStream_t st = as_stream(stream);
#define LQ_LAUNCH(NB, slot)                                                                                                     \
    do {                                                                                                                        \
        auto kern = latent_query_kernel<NB>;                                                                                    \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                    \
        CMLB_CUDA(launch_chain(kern, grid, dim3(LQ_THREADS), smem, 1, st, *a, (const __nv_bfloat16*)d_wukt, d_proj, ld, d_row_pos, d_row_slot, rows, (__half*)d_q_f16)); \
    } while (0)
    if (nb == 1) LQ_LAUNCH(1, 0);
    else if (nb == 2) LQ_LAUNCH(2, 1);
    else LQ_LAUNCH(4, 2);
#undef LQ_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_latent_output(const cmlb200_latent* a, const uint16_t* d_wuv, const uint16_t* d_o_bf16, const float* d_proj, int ld, int rows,
                                     uint16_t* d_out_bf16, int out_ld, void* stream) {
    const int rc = check_latent(a, ld, "cmlb200_latent_output");
    if (rc) return rc;
    CMLB_REQUIRE(d_wuv && d_o_bf16 && d_proj && d_out_bf16 && rows > 0 && rows <= 65535 * LQ_ROWS && out_ld >= a->heads * a->vdim, "cmlb200_latent_output: bad argument");
    CMLB_REQUIRE((((uintptr_t)d_wuv | (uintptr_t)d_o_bf16) & 15) == 0, "cmlb200_latent_output: alignment");
    const dim3 grid((a->vdim + 15) / 16, a->heads, (rows + LQ_ROWS - 1) / LQ_ROWS);
    cudaStream_t st = as_stream(stream);
#define LO_LAUNCH(NB) CMLB_CUDA(launch_chain(latent_output_kernel<NB>, grid, dim3(LO_WARPS * 32), 0, 1, st, *a, (const __nv_bfloat16*)d_wuv, (const __nv_bfloat16*)d_o_bf16, d_proj, ld, rows, (__nv_bfloat16*)d_out_bf16, out_ld))
    if (rows <= 8) LO_LAUNCH(1);
    else if (rows <= 16) LO_LAUNCH(2);
    else LO_LAUNCH(4);
#undef LO_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_latent_gather(const cmlb200_latent* a, const int (*keys)[4], int n, uint16_t* d_c_bf16, const cmlb200_attn* s, void* stream) {
    CMLB_REQUIRE(a && keys && n > 0 && n <= 16 && d_c_bf16 && s && s->k_pool && s->block_table, "cmlb200_latent_gather: bad argument");
    CMLB_REQUIRE(a->cache_dtype == CMLB200_DT_F16 && s->block_size == a->block_size && s->kv_heads == a->heads && s->dim == a->dim + a->rot_dim && s->dim_ld >= s->dim,
                 "cmlb200_latent_gather: shapes do not fit");
    GatherList list = {};
    int most = 0;
    for (int i = 0; i < n; i++) {
        CMLB_REQUIRE(keys[i][0] >= 0 && keys[i][1] >= 0 && keys[i][2] > 0 && keys[i][3] >= 0 && keys[i][1] % a->block_size == 0 && keys[i][3] % a->block_size == 0,
                     "cmlb200_latent_gather: range %d", i);
        list.k[i] = make_int4(keys[i][0], keys[i][1], keys[i][2], keys[i][3]);
        if (keys[i][2] > most) most = keys[i][2];
    }
    const dim3 grid((most + a->block_size - 1) / a->block_size, n, a->heads < 8 ? a->heads : 8);
    const bool vec = a->rank % 8 == 0 && a->rot_dim % 8 == 0 && a->dim % 8 == 0 && s->dim_ld % 8 == 0 && (((uintptr_t)d_c_bf16 | (uintptr_t)s->k_pool | (uintptr_t)a->pool) & 15) == 0;
#define LG_LAUNCH(V) CMLB_CUDA(launch_chain(latent_gather_kernel<V>, grid, dim3(256), 0, 1, as_stream(stream), *a, list, (__nv_bfloat16*)d_c_bf16, (__half*)s->k_pool, s->dim_ld, const_cast<int*>(s->block_table), s->table_ld))
    if (vec) LG_LAUNCH(true);
    else LG_LAUNCH(false);
#undef LG_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_latent_query_f32(const cmlb200_latent* a, const float* d_wukt, const float* d_proj, int ld, const int* d_row_pos, const int* d_row_slot,
                                        int rows, float* d_q, void* stream) {
    const int rc = check_latent(a, ld, "cmlb200_latent_query_f32");
    if (rc) return rc;
    CMLB_REQUIRE(d_wukt && d_proj && d_row_pos && d_row_slot && rows > 0 && rows <= 65535 && d_q && a->cache_dtype == CMLB200_DT_F32, "cmlb200_latent_query_f32: bad argument");
    cudaStream_t st = as_stream(stream);
    const int kd = a->rank + a->rot_dim;
    CMLB_CUDA(launch_chain(latent_append_kernel<float>, dim3(rows), dim3(256), (size_t)a->rot_dim * 4, 1, st, *a, const_cast<float*>(d_proj), ld, d_row_pos, d_row_slot,
                           d_q, (size_t)a->heads * kd, kd, a->rank));
    CMLB_CUDA(launch_chain(heads_linear_f32_kernel, dim3((a->rank + 7) / 8, a->heads, rows), dim3(256), 0, 1, st, d_wukt, a->rank, a->dim, d_proj, (size_t)ld,
                           a->dim + a->rot_dim, (const float*)nullptr, (size_t)0, 0, d_q, (size_t)a->heads * kd, kd));
    return CMLB200_OK;
}

extern "C" int cmlb200_latent_output_f32(const cmlb200_latent* a, const float* d_wuv, const float* d_o, const float* d_proj, int ld, int rows, float* d_out,
                                         int out_ld, void* stream) {
    const int rc = check_latent(a, ld, "cmlb200_latent_output_f32");
    if (rc) return rc;
    CMLB_REQUIRE(d_wuv && d_o && d_proj && d_out && rows > 0 && rows <= 65535 && out_ld >= a->heads * a->vdim, "cmlb200_latent_output_f32: bad argument");
    CMLB_CUDA(launch_chain(heads_linear_f32_kernel, dim3((a->vdim + 7) / 8, a->heads, rows), dim3(256), 0, 1, as_stream(stream), d_wuv, a->vdim, a->rank, d_o,
                           (size_t)a->heads * a->rank, a->rank, a->gate_col >= 0 ? d_proj + a->gate_col : (const float*)nullptr, (size_t)ld, a->gate_heads, d_out, (size_t)out_ld, a->vdim));
    return CMLB200_OK;
}
