// Minimal gated recurrence over a step's rows (see cmlb200_gru): per channel S <- (1 - z) S + z c with z = sigmoid of one
// projection and c a piecewise function of another, neither of which looks at the state, so that a portion's recurrence is a
// scan of affine maps. fp32 throughout.
//
//   gru_one_kernel    decoded tokens: a thread per channel
//   gru_rows_kernel   portions: a CTA owns 32 channels of a portion, its 32 warps consecutive shares of the tokens. Each
//                     composes the maps of its share, starts from the composition of those in front, and runs its share again
#include "lm_util.cuh"

namespace {

struct GruIn {
    float z, u, g;
};
__device__ __forceinline__ GruIn gru_load(const cmlb200_gru& a, const float* row, int c) { return {row[a.col + c], row[a.col + a.width + c], row[a.col + 2 * a.width + c]}; }
__device__ __forceinline__ float gru_candidate(float u) { return u >= 0.f ? u + 0.5f : sigmoidf(u); }

template <typename TO>
__global__ void __launch_bounds__(256)
gru_one_kernel(const cmlb200_gru a, const float* __restrict__ proj, int ld, const int* __restrict__ row_pos, const int* __restrict__ row_slot, TO* __restrict__ out, int out_ld) {
    const int c = blockIdx.x * 256 + threadIdx.x, r = blockIdx.y;
    // neither positions and slots nor the states come from the launch in front
    float* state = a.state + (size_t)row_slot[r] * a.width + c;
    float S = c < a.width && row_pos[r] > 0 ? *state : 0.f;
    dep_wait();
    dep_trigger();
    if (c >= a.width) return;
    const GruIn x = gru_load(a, proj + (size_t)r * ld, c);
    const float z = sigmoidf(x.z);
    S = fmaf(z, gru_candidate(x.u), (1.0f - z) * S);
    *state = S;
    out[(size_t)r * out_ld + c] = narrow<TO>(S * silu(x.g));
}

constexpr int GR_WARPS = 32, GR_CHANNELS = 32, GR_AHEAD = 4;

// grid = (channels / 32, portions)
template <typename TO>
__global__ void __launch_bounds__(GR_WARPS * 32)
gru_rows_kernel(const cmlb200_gru a, const float* __restrict__ proj, int ld, const int4* __restrict__ runs, TO* __restrict__ out, int out_ld) {
    __shared__ float mul[GR_WARPS][GR_CHANNELS + 1], add[GR_WARPS][GR_CHANNELS + 1];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = blockIdx.x * GR_CHANNELS + lane;
    dep_wait();
    dep_trigger();
    const int4 run = runs[blockIdx.y];                 // {first row, rows, slot, position}
    const int per = (run.y + GR_WARPS - 1) / GR_WARPS, lo = min(warp * per, run.y), hi = min(lo + per, run.y);
    const bool live = c < a.width;
    const float* row = proj + (size_t)run.x * ld;
    float A = 1.f, B = 0.f;
    if (live)
        for (int i = lo; i < hi; i += GR_AHEAD) {
            float z[GR_AHEAD], u[GR_AHEAD];
#pragma unroll
            for (int k = 0; k < GR_AHEAD; k++) {
                const float* x = row + (size_t)min(i + k, hi - 1) * ld + a.col + c;
                z[k] = x[0];
                u[k] = x[a.width];
            }
#pragma unroll
            for (int k = 0; k < GR_AHEAD; k++) {
                if (i + k >= hi) break;
                const float s = sigmoidf(z[k]), f = 1.0f - s;
                A *= f;
                B = fmaf(s, gru_candidate(u[k]), f * B);
            }
        }
    mul[warp][lane] = A;
    add[warp][lane] = B;
    float* state = a.state + (size_t)run.z * a.width + c;
    float S = live && run.w > 0 ? *state : 0.f;
    __syncthreads();                                   // also: everyone has read the state
    if (!live || lo >= hi) return;
    for (int w = 0; w < warp; w++) S = fmaf(mul[w][lane], S, add[w][lane]);
    for (int i = lo; i < hi; i += GR_AHEAD) {
        GruIn x[GR_AHEAD];
#pragma unroll
        for (int k = 0; k < GR_AHEAD; k++) x[k] = gru_load(a, row + (size_t)min(i + k, hi - 1) * ld, c);
#pragma unroll
        for (int k = 0; k < GR_AHEAD; k++) {
            if (i + k >= hi) break;
            const float z = sigmoidf(x[k].z);
            S = fmaf(z, gru_candidate(x[k].u), (1.0f - z) * S);
            out[(size_t)(run.x + i + k) * out_ld + c] = narrow<TO>(S * silu(x[k].g));
        }
    }
    if (hi == run.y) *state = S;
}

int check_gru(const cmlb200_gru* a, const void* proj, int ld, const void* out, int dtype, int out_ld, const char* who) {
    CMLB_REQUIRE(a && proj && out && a->width > 0 && a->col >= 0 && a->state, "%s: bad argument", who);
    CMLB_REQUIRE(ld >= a->col + 3 * a->width && out_ld >= a->width, "%s: strides %d / %d", who, ld, out_ld);
    CMLB_REQUIRE(dtype == CMLB200_DT_F32 || dtype == CMLB200_DT_BF16, "%s: dtype %d", who, dtype);
    return CMLB200_OK;
}

}  // namespace

extern "C" int cmlb200_gru_one(const cmlb200_gru* a, const float* d_proj, int ld, const int* d_row_pos, const int* d_row_slot, int rows, void* d_out, int out_dtype,
                               int out_ld, void* stream) {
    const int rc = check_gru(a, d_proj, ld, d_out, out_dtype, out_ld, "cmlb200_gru_one");
    if (rc) return rc;
    CMLB_REQUIRE(d_row_pos && d_row_slot && rows > 0 && rows <= 65535, "cmlb200_gru_one: %d rows", rows);
    const dim3 grid((a->width + 255) / 256, rows);
#define GO_LAUNCH(TO) CMLB_CUDA(launch_chain(gru_one_kernel<TO>, grid, dim3(256), 0, 1, as_stream(stream), *a, d_proj, ld, d_row_pos, d_row_slot, (TO*)d_out, out_ld))
    if (out_dtype == CMLB200_DT_BF16) GO_LAUNCH(__nv_bfloat16);
    else GO_LAUNCH(float);
#undef GO_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_gru_rows(const cmlb200_gru* a, const float* d_proj, int ld, const int* d_runs, int runs, void* d_out, int out_dtype, int out_ld, void* stream) {
    const int rc = check_gru(a, d_proj, ld, d_out, out_dtype, out_ld, "cmlb200_gru_rows");
    if (rc) return rc;
    CMLB_REQUIRE(d_runs && runs > 0 && runs <= 65535 && ((uintptr_t)d_runs & 15) == 0, "cmlb200_gru_rows: %d portions", runs);
    const dim3 grid((a->width + GR_CHANNELS - 1) / GR_CHANNELS, runs);
#define GR_LAUNCH(TO) CMLB_CUDA(launch_chain(gru_rows_kernel<TO>, grid, dim3(GR_WARPS * 32), 0, 1, as_stream(stream), *a, d_proj, ld, (const int4*)d_runs, (TO*)d_out, out_ld))
    if (out_dtype == CMLB200_DT_BF16) GR_LAUNCH(__nv_bfloat16);
    else GR_LAUNCH(float);
#undef GR_LAUNCH
    return CMLB200_OK;
}
