// Experts: the router's choice and the plan that orders a step's (row, expert) pairs by expert, the copy of rows into
// that order for the tensor-core product, and the product of the 32-bit path. See cmlb200_moe.
#include "lm_util.cuh"

namespace {

constexpr int ROUTE_WARPS = 8, PLAN_THREADS = 1024;

// The largest of n values above minus infinity (the lower index wins a tie); one warp, the same answer on every lane.
__device__ __forceinline__ int warp_arg_max(const float* v, int n) {
    float best = -INFINITY;
    int at = -1;
    for (int e = threadIdx.x & 31; e < n; e += 32)
        if (v[e] > best) { best = v[e]; at = e; }
    // order-preserving bits; 0: nothing left on this lane
    const unsigned b = __float_as_uint(best), key = at < 0 ? 0u : ((b & 0x80000000u) ? ~b : b | 0x80000000u);
    const unsigned top = __reduce_max_sync(0xffffffffu, key);
    return (int)min(__reduce_min_sync(0xffffffffu, key == top && at >= 0 ? (unsigned)at : 0xffffffffu), (unsigned)n - 1u);
}

// Floats of shared memory a row's choice takes: what is chosen by, the scores, the groups' largest and which are open.
__host__ __device__ inline int route_floats(const cmlb200_moe& m) {
    const int n = m.experts + m.identity;
    return n + (m.correction ? n : 0) + 2 * m.groups;
}

// One warp, one row: softmax over all outputs, or their sigmoids, then `top` times the largest that is left. With a correction the choice
// is by score + correction, otherwise by the sigmoids or by the logits themselves, which have the softmax's order.
__device__ __forceinline__ void route_row(const cmlb200_moe& m, const float* __restrict__ logits, int r, float* z) {
    const int lane = threadIdx.x & 31, n = m.experts + m.identity;
    float* score = m.correction ? z + n : z;                            // without a correction: sigmoids, or still logits
    float mx = -INFINITY, sum = 0.f;
    if (m.sigmoid) {
        for (int e = lane; e < n; e += 32) z[e] = sigmoidf(logits[e]);
    } else {
        for (int e = lane; e < n; e += 32) { const float v = logits[e]; z[e] = v; mx = fmaxf(mx, v); }
        mx = lane_max(mx);
        for (int e = lane; e < n; e += 32) sum += expf(z[e] - mx);
        sum = lane_sum(sum);
    }
    if (m.correction) {
        for (int e = lane; e < n; e += 32) {
            score[e] = m.sigmoid ? z[e] : expf(z[e] - mx) / sum;
            z[e] = score[e] + m.correction[e];
        }
    }
    if (m.groups > 0) {
        float *best = score + n, *open = best + m.groups;
        const int per = n / m.groups;
        __syncwarp();
        for (int g = lane; g < m.groups; g += 32) {
            float one = -INFINITY, two = -INFINITY;
            for (int e = g * per; e < (g + 1) * per; e++) {
                two = fmaxf(two, fminf(one, z[e]));
                one = fmaxf(one, z[e]);
            }
            best[g] = m.group_best == 2 && per > 1 ? one + two : one;
            open[g] = 0.f;
        }
        for (int k = 0; k < m.keep; k++) {
            const int win = warp_arg_max(best, m.groups);
            if (lane == (win & 31)) { best[win] = -INFINITY; open[win] = 1.f; }
        }
        __syncwarp();
        for (int e = lane; e < n; e += 32)
            if (open[e / per] == 0.f) z[e] = -INFINITY;
    }
    float total = 0.f, self = 0.f;
    for (int k = 0; k < m.top; k++) {
        const int win = warp_arg_max(z, n);
        float w = 0.f;
        if (lane == (win & 31)) {
            w = m.correction || m.sigmoid ? score[win] : expf(z[win] - mx) / sum;
            m.ids[r * m.top + k] = win;
            m.weight[r * m.top + k] = w;
            z[win] = -INFINITY;
        }
        w = __shfl_sync(0xffffffffu, w, win & 31);
        total += w;
        if (win >= m.experts) self += w;
    }
    const float f = m.normalize ? m.scale / (total + 1e-20f) : 1.f;
    if (m.normalize) {
        __syncwarp();                                                   // other lanes wrote the weights
        for (int k = lane; k < m.top; k += 32) m.weight[r * m.top + k] *= f;
    }
    if (m.identity > 0 && lane == 0) m.self[r] = self * f;
}

__global__ void __launch_bounds__(ROUTE_WARPS * 32)
route_rows_kernel(const cmlb200_moe m, const float* __restrict__ logits, int ld, int rows) {
    extern __shared__ float z[];
    dep_wait();
    dep_trigger();
    const int warp = threadIdx.x >> 5, r = blockIdx.x * ROUTE_WARPS + warp;
    if (r < rows) route_row(m, logits + (size_t)r * ld, r, z + warp * route_floats(m));
}

// One CTA, with a warp per row where it routes. logits given (up to 32 rows): routes the rows first. Then counts, first positions (multiples of `align`), the
// lists of chosen experts and of row tiles, and a position for every pair.
__global__ void __launch_bounds__(PLAN_THREADS)
plan_kernel(const cmlb200_moe m, const float* __restrict__ logits, int ld, int rows, int align) {
    extern __shared__ float z[];
    int* count = reinterpret_cast<int*>(z);                             // [experts], then the next free position
    dep_wait();
    dep_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pairs = rows * m.top;
    if (logits) {
        if (warp < rows) route_row(m, logits + (size_t)warp * ld, warp, z + warp * route_floats(m));
        __syncthreads();                                                // also orders the choices' global writes for this block
    }
    for (int e = threadIdx.x; e < m.experts; e += blockDim.x) count[e] = 0;
    __syncthreads();
    for (int p = threadIdx.x; p < pairs; p += blockDim.x)
        if (m.ids[p] < m.experts) atomicAdd(&count[m.ids[p]], 1);
    __syncthreads();
    if (warp == 0) {
        int pos = 0, act = 0, til = 0;                                  // positions, chosen experts, tiles so far
        for (int e0 = 0; e0 < m.experts; e0 += 32) {
            const int e = e0 + lane, c = e < m.experts ? count[e] : 0;
            int a = (c + align - 1) / align * align, b = c > 0, t = (c + 127) / 128;
            const int a0 = a, b0 = b, t0 = t;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int x = __shfl_up_sync(0xffffffffu, a, o), y = __shfl_up_sync(0xffffffffu, b, o), w = __shfl_up_sync(0xffffffffu, t, o);
                if (lane >= o) { a += x; b += y; t += w; }
            }
            if (e < m.experts) {
                const int first = pos + a - a0;
                m.start[e] = first;
                m.count[e] = c;
                if (b0) m.active[act + b - 1] = e;
                if (m.tiles)
                    for (int i = 0; i < t0; i++) reinterpret_cast<int4*>(m.tiles)[til + t - t0 + i] = make_int4(first + i * 128, e, min(128, c - i * 128), 0);
                count[e] = first;
            }
            pos += __shfl_sync(0xffffffffu, a, 31);
            act += __shfl_sync(0xffffffffu, b, 31);
            til += __shfl_sync(0xffffffffu, t, 31);
        }
        if (lane == 0) { *m.num_active = act; *m.num_tiles = til; }
    }
    __syncthreads();
    for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
        const int e = m.ids[p];
        if (e >= m.experts) { m.pos[p] = -1; continue; }
        const int at = atomicAdd(&count[e], 1);
        m.pos[p] = at;
        m.src[at] = p / m.top;
        m.expert[at] = e;
    }
}

// xp[pos[pair]] = x[row of the pair], 16 bytes at a time
__global__ void __launch_bounds__(256)
gather_rows_kernel(const cmlb200_moe m, const uint4* __restrict__ x, int ldx, int width, uint4* __restrict__ xp, int ldxp) {
    dep_wait();
    dep_trigger();
    const uint4* s = x + (size_t)blockIdx.x * ldx;
    for (int i = threadIdx.x; i < width; i += 256) {
        const uint4 v = s[i];
        for (int k = 0; k < m.top; k++) {
            const int p = m.pos[blockIdx.x * m.top + k];
            if (p >= 0) xp[(size_t)p * ldxp + i] = v;
        }
    }
}

// 32-bit product: a warp per output value. grid = (columns / 8, rows * top); blockIdx.y counts pairs.
__global__ void __launch_bounds__(256)
moe_linear_f32_kernel(const cmlb200_moe m, const float* __restrict__ W, int ldw, int w_rows, int K, const float* __restrict__ x, int ldx, int gather,
                      int n_out, float* __restrict__ y, int ldy) {
    dep_wait();
    dep_trigger();
    const int p = m.pos[blockIdx.y], n = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (n >= n_out || p < 0) return;
    const float* w = W + ((size_t)m.expert[p] * w_rows + n) * ldw;
    const float* xr = x + (size_t)(gather ? (int)blockIdx.y / m.top : p) * ldx;
    float s = 0.f;
    for (int k = lane; k < K; k += 32) s = fmaf(w[k], xr[k], s);
    s = lane_sum(s);
    if (lane == 0) y[(size_t)p * ldy + n] = s;
}

}  // namespace

extern "C" long cmlb200_moe_positions(int rows, int top, int experts, int align) {
    const long pairs = (long)rows * top, used = pairs < experts ? pairs : experts;
    return pairs + used * (align - 1);
}

extern "C" int cmlb200_moe_route(const cmlb200_moe* m, const float* d_logits, int ld, int rows, int align, void* stream) {
    CMLB_REQUIRE(m && d_logits && rows > 0 && align > 0 && m->experts > 0 && m->top > 0 && m->identity >= 0, "cmlb200_moe_route: bad argument");
    const int outputs = m->experts + m->identity;
    CMLB_REQUIRE(m->top <= outputs && ld >= outputs && (m->identity == 0 || m->self), "cmlb200_moe_route: %d of %d outputs, stride %d", m->top, outputs, ld);
    CMLB_REQUIRE(m->groups == 0 || (m->groups > 0 && outputs % m->groups == 0 && m->keep > 0 && m->keep <= m->groups && m->keep * (outputs / m->groups) >= m->top),
                 "cmlb200_moe_route: %d of %d groups of %d outputs for %d", m->keep, m->groups, outputs, m->top);
    CMLB_REQUIRE(m->group_best >= 0 && m->group_best <= 2, "cmlb200_moe_route: groups by their %d largest", m->group_best);
    CMLB_REQUIRE(m->ids && m->weight && m->pos && m->src && m->expert && m->start && m->count && m->active && m->num_active && m->num_tiles, "cmlb200_moe_route: a plan without arrays");
    CMLB_REQUIRE(outputs <= 1536 && (long)rows * m->top < (1l << 30), "cmlb200_moe_route: %d experts", m->experts);
    cudaStream_t st = as_stream(stream);
    static size_t attr[kMaxDevices] = {};
    static size_t route_attr[kMaxDevices] = {};
    const size_t row = (size_t)route_floats(*m) * 4, counts = (size_t)m->experts * 4;
    const bool fused = rows <= 32 && (size_t)rows * row <= 200 * 1024;
    if (!fused) {
        CMLB_CUDA(cmlb_ensure_smem(route_rows_kernel, ROUTE_WARPS * row, route_attr));
        CMLB_CUDA(launch_chain(route_rows_kernel, dim3((rows + ROUTE_WARPS - 1) / ROUTE_WARPS), dim3(ROUTE_WARPS * 32), ROUTE_WARPS * row, 1, st, *m, d_logits, ld, rows));
    }
    const size_t smem = fused && (size_t)rows * row > counts ? (size_t)rows * row : counts;
    CMLB_CUDA(cmlb_ensure_smem(plan_kernel, smem, attr));
    CMLB_CUDA(launch_chain(plan_kernel, dim3(1), dim3(rows <= 8 ? PLAN_THREADS / 4 : PLAN_THREADS), smem, 1, st, *m, fused ? d_logits : (const float*)nullptr, ld, rows, align));
    return CMLB200_OK;
}

extern "C" int cmlb200_moe_gather(const cmlb200_moe* m, const uint16_t* d_x, int ldx, int rows, int width, uint16_t* d_xp, int ldxp, void* stream) {
    CMLB_REQUIRE(m && d_x && d_xp && rows > 0 && width > 0, "cmlb200_moe_gather: bad argument");
    const int w8 = (width + 7) / 8;
    CMLB_REQUIRE(ldx % 8 == 0 && ldxp % 8 == 0 && ldx >= w8 * 8 && ldxp >= w8 * 8 && (((uintptr_t)d_x | (uintptr_t)d_xp) & 15) == 0, "cmlb200_moe_gather: strides %d / %d", ldx, ldxp);
    CMLB_CUDA(launch_chain(gather_rows_kernel, dim3(rows), dim3(256), 0, 1, as_stream(stream), *m, (const uint4*)d_x, ldx / 8, w8, (uint4*)d_xp, ldxp / 8));
    return CMLB200_OK;
}

extern "C" int cmlb200_moe_linear_f32(const cmlb200_moe* m, const cmlb200_dense* W, const float* d_x, int ldx, int gather, int rows, int n_out, float* d_y,
                                      int ldy, void* stream) {
    CMLB_REQUIRE(m && W && W->w && d_x && d_y && rows > 0, "cmlb200_moe_linear_f32: bad argument");
    CMLB_REQUIRE(W->dtype == CMLB200_DT_F32 && m->experts > 0 && W->rows % m->experts == 0 && n_out > 0 && n_out <= W->rows / m->experts && W->ld >= W->cols &&
                 ldx >= W->cols && ldy >= n_out, "cmlb200_moe_linear_f32: weight [%d, %d], strides %d / %d", W->rows, W->cols, ldx, ldy);
    const int pairs = rows * m->top;
    for (int at = 0; at < pairs; at += 65535 / m->top * m->top) {       // whole rows per launch
        const int n = pairs - at < 65535 / m->top * m->top ? pairs - at : 65535 / m->top * m->top;
        cmlb200_moe part = *m;
        part.pos = m->pos + at;
        CMLB_CUDA(launch_chain(moe_linear_f32_kernel, dim3((n_out + 7) / 8, n), dim3(256), 0, 1, as_stream(stream), part, (const float*)W->w, W->ld,
                               W->rows / m->experts, W->cols, gather ? d_x + (size_t)(at / m->top) * ldx : d_x, ldx, gather, n_out, d_y, ldy));
    }
    return CMLB200_OK;
}
