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

__device__ __forceinline__ void store_pair(float* d, float2 v) { *reinterpret_cast<float2*>(d) = v; }
__device__ __forceinline__ void store_pair(__half* d, float2 v) {
    const __half h[2] = {narrow<__half>(v.x), narrow<__half>(v.y)};
    *reinterpret_cast<uint32_t*>(d) = *reinterpret_cast<const uint32_t*>(h);
}

// grid = (rows, parts). Work is counted in pairs of neighbouring entries of a padded head: queries, keys, values. T: taps where
// they are known (all loads of a pair are then under way together), 0: any number. VEC: heads start at even columns.
template <typename KV, int T, bool VEC>
__global__ void __launch_bounds__(256)
rotate_append_kernel(const cmlb200_attn a, float* __restrict__ qkv, int ld, const int* __restrict__ row_pos, const int* __restrict__ row_slot, int first, int singles,
                     KV* __restrict__ q_out) {
    extern __shared__ float cs[];                      // cosines, then sines, of the row's position
    dep_wait();
    dep_trigger();
    const int r = first + blockIdx.x, p = row_pos[r], slot = row_slot[r], half = a.rot_dims / 2, taps = T ? T : a.taps;
    for (int i = threadIdx.x; i < half; i += 256) sincosf((float)p * a.freq[i], &cs[half + i], &cs[i]);
    int near = 0;                                      // rows directly in front that belong to the same portion
    if (r >= singles)
        while (near < taps - 1 && near < p && r - near - 1 >= singles && row_slot[r - near - 1] == slot) near++;
    __syncthreads();
    const int channels = attn_channels(a), qp = a.heads * (a.dim_ld / 2), kp = a.kv_heads * (a.dim_ld / 2), vp = a.kv_heads * (a.vdim_ld / 2);
    float* row = qkv + (size_t)r * ld;
    float* ring = a.ring + (taps > 0 ? (size_t)slot * taps * channels : 0);
    const size_t at = (size_t)a.block_table[(size_t)slot * a.table_ld + p / a.block_size] * a.block_size + p % a.block_size;
    KV* kd = static_cast<KV*>(a.k_pool) + at * a.kv_heads * a.dim_ld;
    KV* vd = static_cast<KV*>(a.v_pool) + at * a.kv_heads * a.vdim_ld;
    auto load2 = [&](const float* s, int c, bool two) {
        if (VEC) return *reinterpret_cast<const float2*>(s + c);
        return make_float2(s[c], two ? s[c + 1] : 0.f);
    };
    auto convolved = [&](int c, bool two) {
        const float2 now = load2(row, c, two);
        if (taps <= 0) return now;
        float2 y = load2(a.conv + (size_t)(taps - 1) * channels, c, two);
        y.x *= now.x; y.y *= now.y;
#pragma unroll (T ? T : 1)
        for (int t = 1; t < taps; t++) {
            if (t > p) break;
            const float2 w = load2(a.conv + (size_t)(taps - 1 - t) * channels, c, two);
            const float2 x = load2(t <= near ? row - (size_t)t * ld : ring + (size_t)((p - t) % taps) * channels, c, two);
            y.x = fmaf(w.x, x.x, y.x);
            y.y = fmaf(w.y, x.y, y.y);
        }
        if (r < singles) {
            float* d = ring + (size_t)(p % taps) * channels + c;
            d[0] = now.x;
            if (two) d[1] = now.y;
        }
        return y;
    };
    for (int i = blockIdx.y * 256 + threadIdx.x; i < qp + kp + vp; i += gridDim.y * 256) {
        const bool value = i >= qp + kp, query = i < qp;
        const int j = value ? i - qp - kp : (query ? i : i - qp), per = (value ? a.vdim_ld : a.dim_ld) / 2, h = j / per, d = 2 * (j - h * per);
        const int dim = value ? a.vdim : a.dim, c = (value ? (a.heads + a.kv_heads) * a.dim : (query ? 0 : a.heads * a.dim)) + h * dim + d;
        float2 y = make_float2(0.f, 0.f);
        if (d < dim) y = convolved(c, d + 1 < dim);
        if (!value && d < a.rot_dims) {
            const float co = cs[d / 2], si = cs[half + d / 2];
            y = make_float2(y.x * co - y.y * si, y.y * co + y.x * si);
        }
        if (query && !q_out) {
            if (d < dim) row[c] = y.x;
            if (d + 1 < dim) row[c + 1] = y.y;
            continue;
        }
        KV* o = (value ? vd : (query ? q_out + (size_t)r * a.heads * a.dim_ld : kd)) + (size_t)h * 2 * per + d;
        store_pair(o, y);
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
    const int pairs = a->heads * (a->dim_ld / 2) + a->kv_heads * (a->dim_ld / 2 + a->vdim_ld / 2), most = (pairs + 255) / 256;
    int parts = 1;
    while (parts < most && parts * rows < 2 * cmlb_num_sms()) parts++;
    const bool vec = a->dim % 2 == 0 && a->vdim % 2 == 0 && ld % 2 == 0 && (((uintptr_t)d_qkv | (uintptr_t)a->conv | (uintptr_t)a->ring) & 7) == 0;
    const size_t smem = (size_t)a->rot_dims * 4;
#define RA_LAUNCH(KV, T, V) CMLB_CUDA(launch_chain(rotate_append_kernel<KV, T, V>, dim3(rows, parts), dim3(256), smem, 1, as_stream(stream), *a, d_qkv, ld, d_row_pos, d_row_slot, first, singles, (KV*)d_q_out))
#define RA_VEC(KV, T) do { if (vec) RA_LAUNCH(KV, T, true); else RA_LAUNCH(KV, T, false); } while (0)
#define RA_TAPS(KV) do { if (a->taps == 3) RA_VEC(KV, 3); else if (a->taps == 4) RA_VEC(KV, 4); else RA_VEC(KV, 0); } while (0)
    if (a->cache_dtype == CMLB200_DT_F32) RA_TAPS(float);
    else RA_TAPS(__half);
#undef RA_TAPS
#undef RA_VEC
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
