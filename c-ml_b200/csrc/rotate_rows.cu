// Projection rows on their way into attention, for layers that rotate queries and keys and may convolve q, k and v over
// time first (cmlb200_attn with freq, conv): per channel a causal sum over the latest `taps` projections, then the rotation
// of neighbouring entries 2i and 2i + 1 of a head's first rot_dims, then keys and values into the paged cache and queries
// to where the scores read them. Everything is fp32 up to those stores.
//
//   rotate_append_kernel   any rows; a row's earlier projections come from the rows in front of it where they belong to the
//                          same portion, else from the sequence's ring
//   ring_rows_kernel       the last projections of every portion into the rings, once all rows have been read
//
// A ring holds `taps` entries, position p in entry p mod taps. A decoded token reads the entries before its own and
// writes its own, which no other row of the launch looks at; the rows of a portion would overwrite what its first rows still
// read, so theirs are written by a launch of their own.
#include "lm_util.cuh"

namespace {

__device__ __forceinline__ int attn_channels(const cmlb200_attn& a) { return (a.heads + a.kv_heads) * a.dim + a.kv_heads * a.vdim; }

template <int W> struct Cols { float v[W]; };
template <int W, bool VEC> __device__ __forceinline__ Cols<W> load_cols(const float* s, int have) {
    Cols<W> x;
    if constexpr (VEC && W == 4) { const float4 q = *reinterpret_cast<const float4*>(s); x.v[0] = q.x; x.v[1] = q.y; x.v[2] = q.z; x.v[3] = q.w; }
    else
#pragma unroll
        for (int e = 0; e < W; e++) x.v[e] = e < have ? s[e] : 0.f;
    return x;
}
template <int W, bool VEC> __device__ __forceinline__ void store_cols(float* d, const Cols<W>& x, int have) {
    if constexpr (VEC && W == 4) *reinterpret_cast<float4*>(d) = make_float4(x.v[0], x.v[1], x.v[2], x.v[3]);
    else
#pragma unroll
        for (int e = 0; e < W; e++)
            if (e < have) d[e] = x.v[e];
}
// whole padded heads: every store is aligned
template <int W> __device__ __forceinline__ void store_padded(float* d, const Cols<W>& x) {
    if constexpr (W == 4) *reinterpret_cast<float4*>(d) = make_float4(x.v[0], x.v[1], x.v[2], x.v[3]);
    else *reinterpret_cast<float2*>(d) = make_float2(x.v[0], x.v[1]);
}
template <int W> __device__ __forceinline__ void store_padded(__half* d, const Cols<W>& x) {
    __half h[W];
#pragma unroll
    for (int e = 0; e < W; e++) h[e] = narrow<__half>(x.v[e]);
    if constexpr (W == 4) { uint2 u; memcpy(&u, h, sizeof u); *reinterpret_cast<uint2*>(d) = u; }
    else { uint32_t u; memcpy(&u, h, sizeof u); *reinterpret_cast<uint32_t*>(d) = u; }
}

// grid = (groups of R rows, parts). A thread owns W neighbouring entries of a padded head (queries, keys, values in turn) and takes them
// through the group's rows, whose taps it loads once and whose latest projections it keeps. T: taps where they are known, 0: any
// number. VEC: heads and rows start at multiples of four columns.
template <typename KV, int T, bool VEC, int R>
__global__ void __launch_bounds__(256)
rotate_append_kernel(const cmlb200_attn a, float* __restrict__ qkv, int ld, const int* __restrict__ row_pos, const int* __restrict__ row_slot, int first, int rows,
                     int singles, KV* __restrict__ q_out) {
    constexpr int W = VEC ? 4 : 2;
    extern __shared__ float cs[];                      // per row cosines, then sines, of its position
    __shared__ int s_pos[R], s_slot[R], s_near[R], s_at[R];
    dep_wait();
    dep_trigger();
    const int r0 = first + blockIdx.x * R, nr = min(R, first + rows - r0), half = a.rot_dims / 2, taps = T ? T : a.taps;
    for (int i = threadIdx.x; i < nr * half; i += 256) {
        const int k = i / half, j = i - k * half;
        sincosf((float)row_pos[r0 + k] * a.freq[j], &cs[k * a.rot_dims + half + j], &cs[k * a.rot_dims + j]);
    }
    if ((int)threadIdx.x < nr) {
        const int r = r0 + threadIdx.x, p = row_pos[r], slot = row_slot[r];
        int near = 0;                                  // rows directly in front that belong to the same portion
        if (r >= singles)
            while (near < taps - 1 && near < p && r - near - 1 >= singles && row_slot[r - near - 1] == slot) near++;
        s_pos[threadIdx.x] = p;
        s_slot[threadIdx.x] = slot;
        s_near[threadIdx.x] = near;
        s_at[threadIdx.x] = a.block_table[(size_t)slot * a.table_ld + p / a.block_size] * a.block_size + p % a.block_size;
    }
    __syncthreads();
    const int channels = attn_channels(a), qu = a.heads * (a.dim_ld / W), ku = a.kv_heads * (a.dim_ld / W), vu = a.kv_heads * (a.vdim_ld / W);
    for (int i = blockIdx.y * 256 + threadIdx.x; i < qu + ku + vu; i += gridDim.y * 256) {
        const bool value = i >= qu + ku, query = i < qu;
        const int j = value ? i - qu - ku : (query ? i : i - qu), per = (value ? a.vdim_ld : a.dim_ld) / W, h = j / per, d = W * (j - h * per);
        const int dim = value ? a.vdim : a.dim, c = (value ? (a.heads + a.kv_heads) * a.dim : (query ? 0 : a.heads * a.dim)) + h * dim + d, have = min(W, dim - d);
        constexpr int TT = T ? T : 1;
        Cols<W> w[TT];                                 // weight of the token t back
        if (T && have > 0)
#pragma unroll
            for (int t = 0; t < TT; t++) w[t] = load_cols<W, VEC>(a.conv + (size_t)(taps - 1 - t) * channels + c, have);
        Cols<W> rows_now[R];                           // all under way together
        if (have > 0)
#pragma unroll
            for (int k = 0; k < R; k++)
                if (k < nr) rows_now[k] = load_cols<W, VEC>(qkv + (size_t)(r0 + k) * ld + c, have);
#pragma unroll
        for (int k = 0; k < R; k++) {
            if (k >= nr) break;
            const int p = s_pos[k], near = s_near[k], r = r0 + k;
            float* row = qkv + (size_t)r * ld;
            float* ring = a.ring + (taps > 0 ? (size_t)s_slot[k] * taps * channels : 0);
            Cols<W> y;
#pragma unroll
            for (int e = 0; e < W; e++) y.v[e] = 0.f;
            if (have > 0) {
                const Cols<W> now = rows_now[k];
                auto before = [&](int t) { return load_cols<W, VEC>(t <= near ? row - (size_t)t * ld + c : ring + (size_t)((p - t) % taps) * channels + c, have); };
                auto weigh = [&](const Cols<W>& f, const Cols<W>& x) {
#pragma unroll
                    for (int e = 0; e < W; e++) y.v[e] = fmaf(f.v[e], x.v[e], y.v[e]);
                };
                if constexpr (T > 0) {
                    weigh(w[0], now);
#pragma unroll
                    for (int t = 1; t < T; t++) {
                        if (t <= near && t <= k) weigh(w[t], rows_now[k >= t ? k - t : 0]);
                        else if (t <= p) weigh(w[t], before(t));
                    }
                } else if (taps > 0) {
                    weigh(load_cols<W, VEC>(a.conv + (size_t)(taps - 1) * channels + c, have), now);
                    for (int t = 1; t < taps && t <= p; t++) weigh(load_cols<W, VEC>(a.conv + (size_t)(taps - 1 - t) * channels + c, have), before(t));
                } else {
                    y = now;
                }
                if (taps > 0 && r < singles) store_cols<W, VEC>(ring + (size_t)(p % taps) * channels + c, now, have);
            }
            if (!value) {
                const float* turn = cs + k * a.rot_dims;
#pragma unroll
                for (int e = 0; e < W; e += 2) {
                    if (d + e >= a.rot_dims) continue;
                    const float co = turn[(d + e) / 2], si = turn[half + (d + e) / 2], u = y.v[e], v = y.v[e + 1];
                    y.v[e] = u * co - v * si;
                    y.v[e + 1] = v * co + u * si;
                }
            }
            if (query && !q_out) {
                if (have > 0) store_cols<W, VEC>(row + c, y, have);      // nothing lies between the heads there
                continue;
            }
            store_padded<W>(value ? static_cast<KV*>(a.v_pool) + ((size_t)s_at[k] * a.kv_heads + h) * a.vdim_ld + d
                                  : (query ? q_out + ((size_t)r * a.heads + h) * a.dim_ld + d : static_cast<KV*>(a.k_pool) + ((size_t)s_at[k] * a.kv_heads + h) * a.dim_ld + d), y);
        }
    }
}

// grid = (portions, taps - 1, parts)
__global__ void __launch_bounds__(256)
ring_rows_kernel(const cmlb200_attn a, const float* __restrict__ qkv, int ld, const int4* __restrict__ runs) {
    dep_wait();
    dep_trigger();
    const int4 run = runs[blockIdx.x];                 // {first row, rows, slot, position}
    const int back = blockIdx.y, channels = attn_channels(a);
    if (back >= run.y) return;
    const float* src = qkv + (size_t)(run.x + run.y - 1 - back) * ld;
    float* dst = a.ring + ((size_t)run.z * a.taps + (run.w + run.y - 1 - back) % a.taps) * channels;
    for (int c = blockIdx.z * 256 + threadIdx.x; c < channels; c += gridDim.z * 256) dst[c] = src[c];
}

int check_rotated(const cmlb200_attn* a, int ld, const char* who) {
    const int rc = cmlb200_attn_check_(a, who);
    if (rc) return rc;
    CMLB_REQUIRE(a->rot_dims >= 0 && a->rot_dims % 2 == 0 && a->rot_dims <= a->dim && (a->rot_dims == 0 || a->freq), "%s: %d of %d dimensions rotated", who, a->rot_dims, a->dim);
    CMLB_REQUIRE(a->taps >= 0 && a->taps <= 64 && (a->taps == 0 || (a->conv && a->ring)), "%s: convolution of %d taps", who, a->taps);
    CMLB_REQUIRE(!a->q_norm && !a->k_norm && !a->keys_as_values, "%s: neither norms nor keys that double as values", who);
    CMLB_REQUIRE(ld >= (a->heads + a->kv_heads) * a->dim + a->kv_heads * a->vdim, "%s: row stride %d", who, ld);
    return CMLB200_OK;
}

}  // namespace

extern "C" int cmlb200_rotate_append(const cmlb200_attn* a, float* d_qkv, int ld, const int* d_row_pos, const int* d_row_slot, int first, int rows, int singles,
                                     void* d_q_out, void* stream) {
    static const char* who = "cmlb200_rotate_append";
    CMLB_REQUIRE(a && d_qkv && d_row_pos && d_row_slot && first >= 0 && rows > 0 && singles >= 0, "%s: bad argument", who);
    const int rc = check_rotated(a, ld, who);
    if (rc) return rc;
    CMLB_REQUIRE(a->taps == 0 || d_q_out, "%s: convolved queries go to rows of their own", who);
    const bool vec = a->dim % 4 == 0 && a->vdim % 4 == 0 && ld % 4 == 0 && (((uintptr_t)d_qkv | (uintptr_t)a->conv | (uintptr_t)a->ring | (uintptr_t)d_q_out) & 15) == 0;
    const int units = (a->heads + a->kv_heads) * (a->dim_ld / (vec ? 4 : 2)) + a->kv_heads * (a->vdim_ld / (vec ? 4 : 2)), most = (units + 255) / 256;
    const int group = rows >= 64 ? 8 : 1, groups = (rows + group - 1) / group;
    int parts = 1;
    while (parts < most && parts * groups < 4 * cmlb_num_sms()) parts++;
    const size_t smem = (size_t)group * a->rot_dims * 4;
#define RA_LAUNCH(KV, T, V, R) CMLB_CUDA(launch_chain(rotate_append_kernel<KV, T, V, R>, dim3(groups, parts), dim3(256), smem, 1, as_stream(stream), *a, d_qkv, ld, d_row_pos, d_row_slot, first, rows, singles, (KV*)d_q_out))
#define RA_ROWS(KV, T, V) do { if (group == 8) RA_LAUNCH(KV, T, V, 8); else RA_LAUNCH(KV, T, V, 1); } while (0)
#define RA_VEC(KV, T) do { if (vec) RA_ROWS(KV, T, true); else RA_ROWS(KV, T, false); } while (0)
#define RA_TAPS(KV) do { if (a->taps == 3) RA_VEC(KV, 3); else if (a->taps == 4) RA_VEC(KV, 4); else RA_VEC(KV, 0); } while (0)
    if (a->cache_dtype == CMLB200_DT_F32) RA_TAPS(float);
    else RA_TAPS(__half);
#undef RA_TAPS
#undef RA_VEC
#undef RA_ROWS
#undef RA_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_ring_rows(const cmlb200_attn* a, const float* d_qkv, int ld, const int* d_runs, int runs, void* stream) {
    static const char* who = "cmlb200_ring_rows";
    CMLB_REQUIRE(a && d_qkv && d_runs && runs > 0, "%s: bad argument", who);
    const int rc = check_rotated(a, ld, who);
    if (rc) return rc;
    CMLB_REQUIRE(((uintptr_t)d_runs & 15) == 0, "%s: the list of portions must be 16-byte aligned", who);
    if (a->taps < 2) return CMLB200_OK;
    const int channels = (a->heads + a->kv_heads) * a->dim + a->kv_heads * a->vdim;
    CMLB_CUDA(launch_chain(ring_rows_kernel, dim3(runs, a->taps - 1, (channels + 1023) / 1024), dim3(256), 0, 1, as_stream(stream), *a, d_qkv, ld, (const int4*)d_runs));
    return CMLB200_OK;
}
