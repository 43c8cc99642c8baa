// Row-wise kernels of the layered models: embedding with a sinusoidal position vector or into residual streams, the
// fused "norm a sublayer's output, add it to the residual, norm the sum for the next sublayer" step and its likes over
// streams and for two sublayers that join together through gates, the
// query/key norm with query temperature and paged cache append, and the gated activation of the
// 32-bit path. The residual and every norm are fp32; the operand handed to the next matrix product
// is bf16 or fp32.
#include "lm_util.cuh"

namespace {

// x[r][s] = scale * table[token[r]] for every stream s. W: 4 or 1 columns at a time.
template <typename T, int W>
__global__ void __launch_bounds__(256)
embed_streams_kernel(const T* __restrict__ table, const int* __restrict__ tokens, float scale, int streams, int width, int vocab, float* __restrict__ x) {
    dep_wait();
    dep_trigger();
    const int r = blockIdx.x;
    int t = tokens[r];
    if (t < 0 || t >= vocab) t = 0;
    const T* src = table + (size_t)t * width;
    float* dst = x + (size_t)r * streams * width;
    for (int i = (blockIdx.y * 256 + threadIdx.x) * W; i < width; i += gridDim.y * 256 * W) {
        if constexpr (W == 4) {
            float4 v;
            if constexpr (sizeof(T) == 4) v = *reinterpret_cast<const float4*>(src + i);
            else {
                const uint2 b = *reinterpret_cast<const uint2*>(src + i);
                v = make_float4(__uint_as_float(b.x << 16), __uint_as_float(b.x & 0xffff0000u), __uint_as_float(b.y << 16), __uint_as_float(b.y & 0xffff0000u));
            }
            v.x *= scale; v.y *= scale; v.z *= scale; v.w *= scale;
            for (int s = 0; s < streams; s++) *reinterpret_cast<float4*>(dst + (size_t)s * width + i) = v;
        } else {
            const float v = widen(src[i]) * scale;
            for (int s = 0; s < streams; s++) dst[(size_t)s * width + i] = v;
        }
    }
}

// One CTA per output row of residual streams. y: the sublayer's output y[r], or the weighted sum of the rows its pairs point
// at, plus the row itself times self_w (identity experts), plus a further row. With y: x_t <- sum_s mix[s][t] x_s + out[t] y.
// With w_next: out = norm(sum_s in[s] x_s) * w_next, whose row waits in shared memory between the passes. W: 4 or 1 columns
// at a time; a thread meets the same columns in every pass, so `out` may be the rows h that identity experts return.
template <typename TO, int S, int W>
__global__ void __launch_bounds__(S <= 2 ? 1024 : 512)
stream_join_kernel(const cmlb200_streams hc, float* __restrict__ x, const float* __restrict__ y, int ldy, int parts, const int* __restrict__ part_pos,
                   const float* __restrict__ part_w, const float* __restrict__ self_w, const TO* h, const float* __restrict__ add, int ld_add,
                   const float* __restrict__ w_next, float eps, int width, const int* __restrict__ idx, TO* out, int ldo) {
    extern __shared__ __align__(16) float row[];
    __shared__ float red[32];
    float mix[S][S], to[S], from[S];
#pragma unroll
    for (int s = 0; s < S; s++) {
        const bool have = s < hc.streams;
        from[s] = have ? (hc.in ? hc.in[s] : 1.f) : 0.f;
        to[s] = y && have ? hc.out[s] : 0.f;
#pragma unroll
        for (int t = 0; t < S; t++) mix[s][t] = y && have && t < hc.streams ? hc.mix[s * hc.streams + t] : 0.f;
    }
    dep_wait();
    dep_trigger();
    const int r = blockIdx.x;
    float* xr = x + (size_t)(idx ? idx[r] : r) * hc.streams * width;
    const float own = self_w ? self_w[r] : 0.f;
    auto load = [](const float* p, float (&v)[W]) {
        if constexpr (W == 4) { const float4 q = *reinterpret_cast<const float4*>(p); v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w; }
        else v[0] = *p;
    };
    auto store = [](float* p, const float (&v)[W]) {
        if constexpr (W == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        else *p = v[0];
    };
    float ss = 0.f;
    for (int i = threadIdx.x * W; i < width; i += blockDim.x * W) {
        float v[S][W], u[W];
#pragma unroll
        for (int s = 0; s < S; s++)
            if (s < hc.streams) load(xr + (size_t)s * width + i, v[s]);
            else
#pragma unroll
                for (int e = 0; e < W; e++) v[s][e] = 0.f;
#pragma unroll
        for (int e = 0; e < W; e++) u[e] = 0.f;
        if (y) {
            float z[W], p[W];
#pragma unroll
            for (int e = 0; e < W; e++) z[e] = 0.f;
            if (parts > 0) {
#pragma unroll 4
                for (int k = 0; k < parts; k++) {
                    const int at = part_pos[r * parts + k];
                    if (at < 0) continue;
                    const float w = part_w[r * parts + k];
                    load(y + (size_t)at * ldy + i, p);
#pragma unroll
                    for (int e = 0; e < W; e++) z[e] = fmaf(w, p[e], z[e]);
                }
            } else {
                load(y + (size_t)r * ldy + i, z);
            }
            if (own != 0.f)
#pragma unroll
                for (int e = 0; e < W; e++) z[e] = fmaf(own, widen(h[(size_t)r * ldo + i + e]), z[e]);
            if (add) {
                load(add + (size_t)r * ld_add + i, p);
#pragma unroll
                for (int e = 0; e < W; e++) z[e] += p[e];
            }
#pragma unroll
            for (int t = 0; t < S; t++) {
                if (t >= hc.streams) continue;
                float n[W];
#pragma unroll
                for (int e = 0; e < W; e++) {
                    n[e] = to[t] * z[e];
#pragma unroll
                    for (int s = 0; s < S; s++) n[e] = fmaf(mix[s][t], v[s][e], n[e]);
                    u[e] = fmaf(from[t], n[e], u[e]);
                }
                store(xr + (size_t)t * width + i, n);
            }
        } else {
#pragma unroll
            for (int s = 0; s < S; s++)
#pragma unroll
                for (int e = 0; e < W; e++) u[e] = fmaf(from[s], v[s][e], u[e]);
        }
        store(row + i, u);
#pragma unroll
        for (int e = 0; e < W; e++) ss = fmaf(u[e], u[e], ss);
    }
    if (!w_next) return;
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
    TO* o = out + (size_t)r * ldo;
    for (int i = threadIdx.x * W; i < width; i += blockDim.x * W) {
        float v[W], w[W];
        load(row + i, v);
        load(w_next + i, w);
        TO n[W];
#pragma unroll
        for (int e = 0; e < W; e++) n[e] = narrow<TO>(v[e] * inv * w[e]);
        if constexpr (W == 4 && sizeof(TO) == 2) {
            uint2 b;
            memcpy(&b, n, sizeof b);
            *reinterpret_cast<uint2*>(o + i) = b;
        } else if constexpr (W == 4) {
            store(reinterpret_cast<float*>(o + i), reinterpret_cast<const float(&)[W]>(n));
        } else {
            o[i] = n[0];
        }
    }
}

// One CTA per row. m: j.a, or half the sum of the norms of j.a and j.b; f: a row, or the weighted sum of the rows its pairs point at.
// x += sigmoid(ga) m + sigmoid(gf) f (+ table[token]); with w_next: out = norm(x) * w_next, whose row waits in shared memory.
// W: 4 or 1 columns at a time.
template <typename TO, typename TE, int W>
__global__ void __launch_bounds__(1024)
gated_join_kernel(const cmlb200_gated_join j, int parts, const int* __restrict__ part_pos, const float* __restrict__ part_w, float* __restrict__ x,
                  const float* __restrict__ w_next, float eps, int width, TO* __restrict__ out, int ldo) {
    extern __shared__ __align__(16) float row[];
    __shared__ float red[32];
    __shared__ float2 red2[32];
    dep_wait();
    dep_trigger();
    const int r = blockIdx.x;
    const float *a = j.a + (size_t)r * j.ldm, *b = j.b ? j.b + (size_t)r * j.ldm : nullptr;
    const float *ga = j.ga + (size_t)r * j.ldg, *gf = j.f ? j.gf + (size_t)r * j.ldg : nullptr;
    float* xr = x + (size_t)r * width;
    const TE* again = nullptr;
    if (j.table) {
        const int t = j.tokens[r];
        again = static_cast<const TE*>(j.table) + (size_t)(t < 0 || t >= j.vocab ? 0 : t) * width;
    }
    auto load = [](const float* p, float (&v)[W]) {
        if constexpr (W == 4) { const float4 q = *reinterpret_cast<const float4*>(p); v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w; }
        else v[0] = *p;
    };
    auto store = [](float* p, const float (&v)[W]) {
        if constexpr (W == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        else *p = v[0];
    };
    float ia = 1.f, ib = 1.f;
    if (b) {
        const float2 ss = block_sum2(square_share(a, width), square_share(b, width), red2);
        ia = 0.5f / sqrtf(ss.x / (float)width + eps);
        ib = 0.5f / sqrtf(ss.y / (float)width + eps);
    }
    float ss = 0.f;
    for (int i = threadIdx.x * W; i < width; i += blockDim.x * W) {
        float v[W], m[W], g[W], p[W];
        load(xr + i, v);
        load(a + i, m);
        load(ga + i, g);
        if (b) {
            float wa[W], wb[W];
            load(b + i, p);
            load(j.a_norm + i, wa);
            load(j.b_norm + i, wb);
#pragma unroll
            for (int e = 0; e < W; e++) m[e] = m[e] * ia * wa[e] + p[e] * ib * wb[e];
        }
#pragma unroll
        for (int e = 0; e < W; e++) v[e] = fmaf(sigmoidf(g[e]), m[e], v[e]);
        if (j.f) {
            if (parts > 0) {
#pragma unroll
                for (int e = 0; e < W; e++) m[e] = 0.f;
#pragma unroll 4
                for (int k = 0; k < parts; k++) {
                    const float w = part_w[r * parts + k];
                    load(j.f + (size_t)part_pos[r * parts + k] * j.ldf + i, p);
#pragma unroll
                    for (int e = 0; e < W; e++) m[e] = fmaf(w, p[e], m[e]);
                }
            } else {
                load(j.f + (size_t)r * j.ldf + i, m);
            }
            load(gf + i, g);
#pragma unroll
            for (int e = 0; e < W; e++) v[e] = fmaf(sigmoidf(g[e]), m[e], v[e]);
        }
        if (again)
#pragma unroll
            for (int e = 0; e < W; e++) v[e] += widen(again[i + e]);
        store(xr + i, v);
        store(row + i, v);
#pragma unroll
        for (int e = 0; e < W; e++) ss = fmaf(v[e], v[e], ss);
    }
    if (!w_next) return;
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
    TO* o = out + (size_t)r * ldo;
    for (int i = threadIdx.x * W; i < width; i += blockDim.x * W) {
        float v[W], w[W];
        load(row + i, v);
        load(w_next + i, w);
        TO n[W];
#pragma unroll
        for (int e = 0; e < W; e++) n[e] = narrow<TO>(v[e] * inv * w[e]);
        if constexpr (W == 4 && sizeof(TO) == 2) {
            uint2 q;
            memcpy(&q, n, sizeof q);
            *reinterpret_cast<uint2*>(o + i) = q;
        } else if constexpr (W == 4) {
            store(reinterpret_cast<float*>(o + i), reinterpret_cast<const float(&)[W]>(n));
        } else {
            o[i] = n[0];
        }
    }
}

// out[r] = norm of columns col .. col + n - 1 of row r, times w
template <typename TO>
__global__ void __launch_bounds__(256)
norm_columns_kernel(const float* __restrict__ x, int ld, int col, int n, const float* __restrict__ w, float eps, TO* __restrict__ out, int ldo) {
    __shared__ float red[32];
    dep_wait();
    dep_trigger();
    const float* src = x + (size_t)blockIdx.x * ld + col;
    const float inv = 1.0f / sqrtf(block_sum(square_share(src, n), red) / (float)n + eps);
    for (int i = threadIdx.x; i < n; i += 256) out[(size_t)blockIdx.x * ldo + i] = narrow<TO>(src[i] * inv * w[i]);
}

__global__ void __launch_bounds__(256)
act_rows_f32_kernel(const float* __restrict__ z, int ld, int ff, int act, float* __restrict__ f, int ldf) {
    dep_wait();
    dep_trigger();
    for (int c = blockIdx.y * 256 + threadIdx.x; c < ff; c += gridDim.y * 256) f[(size_t)blockIdx.x * ldf + c] = unary_act(act, z[(size_t)blockIdx.x * ld + c]);
}

__global__ void __launch_bounds__(256)
pack_columns_kernel(const float* __restrict__ x, int ld, int col, int n, int more, int at, __nv_bfloat16* __restrict__ out, int ldo) {
    dep_wait();
    dep_trigger();
    const float* src = x + (size_t)blockIdx.x * ld + col;
    for (int i = threadIdx.x; i < n + more; i += 256) out[(size_t)blockIdx.x * ldo + (i < n ? i : at + i - n)] = __float2bfloat16_rn(src[i]);
}

// x[r] = table[token[r]] (+ the position vector: entry 2i = sin(p f_i), entry 2i + 1 = cos(p f_i),
// f_i = freq[i], angle and sine in fp32). freq == NULL: no position vector.
template <typename T>
__global__ void __launch_bounds__(256)
embed_rows_kernel(const T* __restrict__ table, const int* __restrict__ tokens, const int* __restrict__ pos, const float* __restrict__ freq,
                  int width, int vocab, float* __restrict__ x) {
    dep_wait();
    dep_trigger();
    const int r = blockIdx.x;
    int t = tokens[r];
    if (t < 0 || t >= vocab) t = 0;
    const float p = (float)pos[r];
    const T* src = table + (size_t)t * width;
    float* dst = x + (size_t)r * width;
    for (int i = blockIdx.y * 256 + threadIdx.x; 2 * i < width; i += gridDim.y * 256) {
        float s = 0.f, c = 0.f;
        if (freq) sincosf(p * freq[i], &s, &c);
        dst[2 * i] = widen(src[2 * i]) + s;
        if (2 * i + 1 < width) dst[2 * i + 1] = widen(src[2 * i + 1]) + c;
    }
}

// One CTA per output row. y == NULL: out = norm(x[idx]) * w_next. Otherwise x += norm(y) * w_post
// (w_post == NULL: x += y) and, when w_next is given, out = norm(x) * w_next; raw: out = x. The row stays in
// shared memory between the passes. Columns dim .. ldo of `out` are left alone. PARTS: row r of y is the sum of the rows
// part_pos[r * parts + k] with weights part_w[r * parts + k].
template <typename TO, bool VEC, bool PARTS>
__global__ void __launch_bounds__(1024)
residual_norm_kernel(float* __restrict__ x, const float* __restrict__ y, int ldy, const float* __restrict__ w_post,
                     const float* __restrict__ w_next, float eps, int dim, const int* __restrict__ idx, TO* __restrict__ out, int ldo, int raw,
                     int parts, const int* __restrict__ part_pos, const float* __restrict__ part_w) {
    extern __shared__ __align__(16) float row[];
    __shared__ float red[32];
    dep_wait();
    dep_trigger();
    const int r = blockIdx.x;
    auto part_sum = [&](auto zero, int i) {
        auto s = zero;
#pragma unroll 4
        for (int k = 0; k < parts; k++) {
            const float w = part_w[r * parts + k];
            const float* p = y + (size_t)part_pos[r * parts + k] * ldy + i;
            if constexpr (sizeof(s) == 16) {
                const float4 v = *reinterpret_cast<const float4*>(p);
                s.x = fmaf(w, v.x, s.x); s.y = fmaf(w, v.y, s.y); s.z = fmaf(w, v.z, s.z); s.w = fmaf(w, v.w, s.w);
            } else {
                s = fmaf(w, *p, s);
            }
        }
        return s;
    };
    float* xr = x + (size_t)(idx ? idx[r] : r) * dim;
    float ss = 0.f;
    if (y) {
        const float* yr = y + (size_t)r * ldy;
        if (VEC) {
            for (int i = threadIdx.x * 4; i < dim; i += blockDim.x * 4) {
                const float4 v = PARTS ? part_sum(make_float4(0.f, 0.f, 0.f, 0.f), i) : *reinterpret_cast<const float4*>(yr + i);
                *reinterpret_cast<float4*>(row + i) = v;
                ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
            }
        } else {
            for (int i = threadIdx.x; i < dim; i += blockDim.x) { const float v = PARTS ? part_sum(0.f, i) : yr[i]; row[i] = v; ss = fmaf(v, v, ss); }
        }
        const float inv = w_post ? 1.0f / sqrtf(block_sum(ss, red) / (float)dim + eps) : 1.0f;
        ss = 0.f;
        if (VEC) {                                      // a thread meets the same columns in every pass
            for (int i = threadIdx.x * 4; i < dim; i += blockDim.x * 4) {
                const float4 a = *reinterpret_cast<const float4*>(xr + i), v = *reinterpret_cast<const float4*>(row + i);
                const float4 w = w_post ? *reinterpret_cast<const float4*>(w_post + i) : make_float4(1.f, 1.f, 1.f, 1.f);
                const float4 o = make_float4(a.x + v.x * inv * w.x, a.y + v.y * inv * w.y, a.z + v.z * inv * w.z, a.w + v.w * inv * w.w);
                *reinterpret_cast<float4*>(xr + i) = o;
                *reinterpret_cast<float4*>(row + i) = o;
                ss = fmaf(o.x, o.x, fmaf(o.y, o.y, fmaf(o.z, o.z, fmaf(o.w, o.w, ss))));
            }
        } else {
            for (int i = threadIdx.x; i < dim; i += blockDim.x) {
                const float o = xr[i] + row[i] * inv * (w_post ? w_post[i] : 1.0f);
                xr[i] = o;
                row[i] = o;
                ss = fmaf(o, o, ss);
            }
        }
    } else if (VEC) {
        for (int i = threadIdx.x * 4; i < dim; i += blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(xr + i);
            *reinterpret_cast<float4*>(row + i) = v;
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        }
    } else {
        for (int i = threadIdx.x; i < dim; i += blockDim.x) { const float v = xr[i]; row[i] = v; ss = fmaf(v, v, ss); }
    }
    if (!w_next && !raw) return;
    const float inv = raw ? 1.0f : 1.0f / sqrtf(block_sum(ss, red) / (float)dim + eps);
    TO* o = out + (size_t)r * ldo;
    if (VEC) {
        for (int i = threadIdx.x * 4; i < dim; i += blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(row + i), w = raw ? make_float4(1.f, 1.f, 1.f, 1.f) : *reinterpret_cast<const float4*>(w_next + i);
            const float a = v.x * inv * w.x, b = v.y * inv * w.y, c = v.z * inv * w.z, d = v.w * inv * w.w;
            if (sizeof(TO) == 2) {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
                *reinterpret_cast<uint2*>(o + i) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
            } else {
                *reinterpret_cast<float4*>(o + i) = make_float4(a, b, c, d);
            }
        }
    } else {
        for (int i = threadIdx.x; i < dim; i += blockDim.x) o[i] = narrow<TO>(raw ? row[i] : row[i] * inv * w_next[i]);
    }
}

// f = a N(z) + b N(z^2) + c N(z^3) + e, N(v) = v / sqrt(mean(v^2) + eps) over the row. One CTA per row.
template <typename TO, bool VEC>
__global__ void __launch_bounds__(1024)
poly_norm_kernel(const float* __restrict__ z, int ld, int ff, const float* __restrict__ coef, float eps, TO* __restrict__ f, int ldf) {
    extern __shared__ __align__(16) float row[];
    __shared__ float red[32];
    __shared__ float2 red2[32];
    const float a = coef[0], b = coef[1], c = coef[2], e = coef[3];
    dep_wait();
    dep_trigger();
    const float* zr = z + (size_t)blockIdx.x * ld;
    float s1 = 0.f, s2 = 0.f, s3 = 0.f;
    auto add = [&](float v) {
        const float q = v * v;
        s1 += q;
        s2 = fmaf(q, q, s2);
        s3 = fmaf(q * q, q, s3);
    };
    if (VEC) {
        for (int i = threadIdx.x * 4; i < ff; i += blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(zr + i);
            *reinterpret_cast<float4*>(row + i) = v;
            add(v.x); add(v.y); add(v.z); add(v.w);
        }
    } else {
        for (int i = threadIdx.x; i < ff; i += blockDim.x) { const float v = zr[i]; row[i] = v; add(v); }
    }
    const float2 t = block_sum2(s1, s2, red2);
    const float n = (float)ff, u = block_sum(s3, red);
    const float i1 = a / sqrtf(t.x / n + eps), i2 = b / sqrtf(t.y / n + eps), i3 = c / sqrtf(u / n + eps);
    auto value = [&](float v) { return fmaf(v, fmaf(v, fmaf(v, i3, i2), i1), e); };
    TO* o = f + (size_t)blockIdx.x * ldf;
    if (VEC) {
        for (int i = threadIdx.x * 4; i < ff; i += blockDim.x * 4) {
            const float4 v = *reinterpret_cast<const float4*>(row + i);
            const TO w[4] = {narrow<TO>(value(v.x)), narrow<TO>(value(v.y)), narrow<TO>(value(v.z)), narrow<TO>(value(v.w))};
            if (sizeof(TO) == 2) *reinterpret_cast<uint2*>(o + i) = *reinterpret_cast<const uint2*>(w);
            else *reinterpret_cast<float4*>(o + i) = *reinterpret_cast<const float4*>(w);
        }
    } else {
        for (int i = threadIdx.x; i < ff; i += blockDim.x) o[i] = narrow<TO>(value(row[i]));
    }
}

// One CTA per row of stacked projections [q | k | v | ..]: q is normed over all of its heads at once,
// multiplied by the temperature of its position and left in place (fp32); k is normed the same way and
// goes with v into the row's cache slot, each head padded with zeros to its stride in the pool.
template <typename KV>
__device__ __forceinline__ void store4(KV* dst, float4 v) {
    if (sizeof(KV) == 4) *reinterpret_cast<float4*>(dst) = v;
    else {
        const KV h[4] = {narrow<KV>(v.x), narrow<KV>(v.y), narrow<KV>(v.z), narrow<KV>(v.w)};
        *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<const uint2*>(h);
    }
}

// VEC: dim and vdim are multiples of 4 and so is the row stride: four elements at a time, none of which
// straddles a head.
template <typename KV, bool VEC>
__global__ void __launch_bounds__(256)
qk_norm_append_kernel(float* __restrict__ qkv, int ld, const int* __restrict__ row_pos, const int* __restrict__ row_slot,
                      const cmlb200_attn a, KV* __restrict__ kpool, KV* __restrict__ vpool) {
    __shared__ float2 red[32];
    extern __shared__ float inv[];                     // head_norm: of every query head, then of every key head
    dep_wait();
    dep_trigger();
    const int r = blockIdx.x, qw = a.heads * a.dim, kw = a.kv_heads * a.dim, vcol = qw + (a.keys_as_values ? 0 : kw);
    float* row = qkv + (size_t)r * ld;
    const int p = row_pos[r];
    const size_t slot = (size_t)a.block_table[(size_t)row_slot[r] * a.table_ld + p / a.block_size] * a.block_size + p % a.block_size;
    const float temp = a.temp_every > 0.f ? 1.0f + a.temp_coef * logf(floorf((float)(p + 1) / a.temp_every) + 1.0f) : 1.0f;
    KV* kd = kpool + slot * a.kv_heads * a.dim_ld;
    KV* vd = vpool + slot * a.kv_heads * a.vdim_ld;
    float2 ss = make_float2(0.f, 0.f);
    if (VEC && a.head_norm && a.dim <= 256) {          // a warp per head, which it holds in registers
        const int lane = threadIdx.x & 31;
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f), ones = make_float4(1.f, 1.f, 1.f, 1.f);
#pragma unroll 4
        for (int j = threadIdx.x >> 5; j < a.heads + a.kv_heads; j += 8) {
            const bool query = j < a.heads;
            const float* norm = query ? a.q_norm : a.k_norm;
            float* v = row + (size_t)j * a.dim;
            float4 x[2];
            float s = 0.f;
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const int d = lane * 4 + 128 * i;
                x[i] = d < a.dim ? *reinterpret_cast<const float4*>(v + d) : zero;
                s = fmaf(x[i].x, x[i].x, fmaf(x[i].y, x[i].y, fmaf(x[i].z, x[i].z, fmaf(x[i].w, x[i].w, s))));
            }
            s = lane_sum(s);
            const float f = (norm ? 1.0f / sqrtf(s / (float)a.dim + a.eps) : 1.0f) * (query ? temp : 1.0f);
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const int d = lane * 4 + 128 * i;
                const float4 w = norm && d < a.dim ? *reinterpret_cast<const float4*>(norm + d) : ones;
                const float4 y = make_float4(x[i].x * f * w.x, x[i].y * f * w.y, x[i].z * f * w.z, x[i].w * f * w.w);
                if (query) {
                    if (d < a.dim) *reinterpret_cast<float4*>(v + d) = y;
                } else if (d < a.dim_ld) {             // zeros behind dim
                    store4(kd + (size_t)(j - a.heads) * a.dim_ld + d, y);
                    if (a.keys_as_values) store4(vd + (size_t)(j - a.heads) * a.vdim_ld + d, x[i]);
                }
            }
        }
        if (!a.keys_as_values)
            for (int i = threadIdx.x * 4; i < a.kv_heads * a.vdim_ld; i += 1024) {
                const int g = i / a.vdim_ld, d = i - g * a.vdim_ld;
                store4(vd + i, d < a.vdim ? *reinterpret_cast<const float4*>(row + vcol + g * a.vdim + d) : zero);
            }
        return;
    }
    if (a.head_norm) {
        const int lane = threadIdx.x & 31;
        for (int j = threadIdx.x >> 5; j < a.heads + a.kv_heads; j += 8) {
            const float* v = row + (size_t)j * a.dim;
            float s = 0.f;
            for (int d = lane; d < a.dim; d += 32) s = fmaf(v[d], v[d], s);
            s = lane_sum(s);
            if (lane == 0) inv[j] = (j < a.heads ? a.q_norm : a.k_norm) ? 1.0f / sqrtf(s / (float)a.dim + a.eps) : 1.0f;
        }
        __syncthreads();
    } else if (a.q_norm || a.k_norm) {
        ss = block_sum2(square_share(row, qw), square_share(row + qw, kw), red);
    }
    const bool same_q = !a.q_norm && a.temp_every <= 0.f;                // q stays as it is
    const float iq = a.q_norm ? 1.0f / sqrtf(ss.x / (float)qw + a.eps) : 1.0f, ik = a.k_norm ? 1.0f / sqrtf(ss.y / (float)kw + a.eps) : 1.0f;
    if (VEC) {
#pragma unroll 4
        for (int i = same_q ? qw : threadIdx.x * 4; i < qw; i += 1024) {
            float4 v = *reinterpret_cast<const float4*>(row + i);
            const int j = a.head_norm ? i / a.dim : 0;
            const float f = a.head_norm ? inv[j] : iq;
            const float4 w = a.q_norm ? *reinterpret_cast<const float4*>(a.q_norm + i - j * a.dim) : make_float4(1.f, 1.f, 1.f, 1.f);
            v.x = v.x * f * w.x * temp; v.y = v.y * f * w.y * temp; v.z = v.z * f * w.z * temp; v.w = v.w * f * w.w * temp;
            *reinterpret_cast<float4*>(row + i) = v;
        }
#pragma unroll 4
        for (int i = threadIdx.x * 4; i < a.kv_heads * a.dim_ld; i += 1024) {
            const int g = i / a.dim_ld, d = i - g * a.dim_ld, c = g * a.dim + d;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (d < a.dim) {
                v = *reinterpret_cast<const float4*>(row + qw + c);
                const float4 w = a.k_norm ? *reinterpret_cast<const float4*>(a.k_norm + (a.head_norm ? d : c)) : make_float4(1.f, 1.f, 1.f, 1.f);
                const float f = a.head_norm ? inv[a.heads + g] : ik;
                v.x *= f * w.x; v.y *= f * w.y; v.z *= f * w.z; v.w *= f * w.w;
            }
            store4(kd + i, v);
        }
#pragma unroll 4
        for (int i = threadIdx.x * 4; i < a.kv_heads * a.vdim_ld; i += 1024) {
            const int g = i / a.vdim_ld, d = i - g * a.vdim_ld;
            store4(vd + i, d < a.vdim ? *reinterpret_cast<const float4*>(row + vcol + g * a.vdim + d) : make_float4(0.f, 0.f, 0.f, 0.f));
        }
        return;
    }
    for (int i = same_q ? qw : threadIdx.x; i < qw; i += 256) {
        const int j = a.head_norm ? i / a.dim : 0;
        row[i] = row[i] * (a.head_norm ? inv[j] : iq) * (a.q_norm ? a.q_norm[i - j * a.dim] : 1.0f) * temp;
    }
    for (int i = threadIdx.x; i < a.kv_heads * a.dim_ld; i += 256) {
        const int g = i / a.dim_ld, d = i - g * a.dim_ld, c = g * a.dim + d;
        kd[i] = narrow<KV>(d < a.dim ? row[qw + c] * (a.head_norm ? inv[a.heads + g] : ik) * (a.k_norm ? a.k_norm[a.head_norm ? d : c] : 1.0f) : 0.f);
    }
    for (int i = threadIdx.x; i < a.kv_heads * a.vdim_ld; i += 256) {
        const int g = i / a.vdim_ld, d = i - g * a.vdim_ld;
        vd[i] = narrow<KV>(d < a.vdim ? row[vcol + g * a.vdim + d] : 0.f);
    }
}

// f[r][c] = act(gate) * up of rows whose columns come in pairs of 16-wide groups (16 gate, 16 up, ..)
__global__ void __launch_bounds__(256)
glu_rows_f32_kernel(const float* __restrict__ gu, int ld, int ff, int act, float limit, float* __restrict__ f, int ldf) {
    dep_wait();
    dep_trigger();
    const float* g = gu + (size_t)blockIdx.x * ld;
    for (int c = blockIdx.y * 256 + threadIdx.x; c < ff; c += gridDim.y * 256) {
        const int b = (c >> 4) * 32 + (c & 15);
        f[(size_t)blockIdx.x * ldf + c] = glu_act(act, g[b], g[b + 16], limit);
    }
}

// The next step of a decode loop that stays on the device: token = the one just picked, position + 1.
__global__ void advance_tokens_kernel(const int* __restrict__ picked, int rows, int* __restrict__ tokens, int* __restrict__ pos, int* __restrict__ hist,
                                      int* __restrict__ step) {
    dep_wait();
    dep_trigger();
    const int s = *step;
    for (int i = threadIdx.x; i < rows; i += blockDim.x) {
        tokens[i] = picked[i];
        pos[i] += 1;
        hist[(size_t)s * rows + i] = picked[i];
    }
    __syncthreads();
    if (threadIdx.x == 0) *step = s + 1;
}

}  // namespace

extern "C" int cmlb200_embed_rows(const void* d_table, int dtype, const int* d_tokens, const int* d_pos, const float* d_freq, int rows, int width,
                                  int vocab, float* d_x, void* stream) {
    CMLB_REQUIRE(d_table && d_tokens && d_pos && d_x && rows > 0 && width > 0 && vocab > 0, "cmlb200_embed_rows: bad argument");
    CMLB_REQUIRE(dtype == CMLB200_DT_F32 || dtype == CMLB200_DT_BF16, "cmlb200_embed_rows: dtype %d", dtype);
    const dim3 grid(rows, rows < 64 ? (width + 511) / 512 : 1);
    cudaStream_t st = as_stream(stream);
    if (dtype == CMLB200_DT_BF16)
        CMLB_CUDA(launch_chain(embed_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, 1, st, (const __nv_bfloat16*)d_table, d_tokens, d_pos, d_freq, width, vocab, d_x));
    else
        CMLB_CUDA(launch_chain(embed_rows_kernel<float>, grid, dim3(256), 0, 1, st, (const float*)d_table, d_tokens, d_pos, d_freq, width, vocab, d_x));
    return CMLB200_OK;
}

static int launch_residual(float* d_x, const float* d_y, int ldy, const cmlb200_moe* parts, const float* d_w_post, const float* d_w_next, float eps,
                           int rows, int dim, const int* d_row_idx, void* d_out, int out_dtype, int ldo, int raw, cudaStream_t st) {
    CMLB_REQUIRE(out_dtype == CMLB200_DT_F32 || out_dtype == CMLB200_DT_BF16, "residual norm: dtype %d", out_dtype);
    const size_t smem = (size_t)((dim + 3) / 4) * 16;
    CMLB_REQUIRE(smem <= 200 * 1024, "residual norm: rows of %d elements do not fit shared memory", dim);
    const bool vec = dim % 4 == 0 && (!d_y || ldy % 4 == 0) && ((!d_w_next && !raw) || ldo % 4 == 0) &&
                     (((uintptr_t)d_x | (uintptr_t)d_y | (uintptr_t)d_w_post | (uintptr_t)d_w_next | (uintptr_t)d_out) & 15) == 0;
    // few rows: enough threads that each meets its row once; many rows: small CTAs, several to an SM
    int threads = 256;
    if (rows <= 2 * cmlb_num_sms()) while (threads < 1024 && threads * 4 < dim) threads *= 2;
    static size_t attr[8][kMaxDevices] = {};
#define RN_LAUNCH(TO, V, P, slot)                                                                                                   \
    do {                                                                                                                            \
        auto kern = residual_norm_kernel<TO, V, P>;                                                                                 \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                        \
        CMLB_CUDA(launch_chain(kern, dim3(rows), dim3(threads), smem, 1, st, d_x, d_y, ldy, d_w_post, d_w_next, eps, dim, d_row_idx, (TO*)d_out, ldo, raw, \
                               parts ? parts->top : 0, (const int*)(parts ? parts->pos : nullptr), (const float*)(parts ? parts->weight : nullptr))); \
    } while (0)
#define RN_VEC(TO, P, slot) do { if (vec) RN_LAUNCH(TO, true, P, slot); else RN_LAUNCH(TO, false, P, slot + 1); } while (0)
    if (out_dtype == CMLB200_DT_BF16) { if (parts) RN_VEC(__nv_bfloat16, true, 0); else RN_VEC(__nv_bfloat16, false, 2); }
    else { if (parts) RN_VEC(float, true, 4); else RN_VEC(float, false, 6); }
#undef RN_VEC
#undef RN_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_residual_norm(float* d_x, const float* d_y, int ldy, const float* d_w_post, const float* d_w_next, float eps, int rows,
                                     int dim, const int* d_row_idx, void* d_out, int out_dtype, int ldo, void* stream) {
    CMLB_REQUIRE(d_x && rows > 0 && dim > 0 && (d_y || d_w_next), "cmlb200_residual_norm: bad argument");
    CMLB_REQUIRE(!d_w_next || (d_out && ldo >= dim), "cmlb200_residual_norm: no output for the normed rows");
    CMLB_REQUIRE(!(d_y && d_row_idx) && (!d_y || ldy >= dim), "cmlb200_residual_norm: a row list goes with the norm-only form");
    return launch_residual(d_x, d_y, ldy, nullptr, d_w_post, d_w_next, eps, rows, dim, d_row_idx, d_out, out_dtype, ldo, 0, as_stream(stream));
}

extern "C" int cmlb200_residual_add(float* d_x, const float* d_y, int ldy, const cmlb200_moe* parts, const float* d_w_post, float eps, int rows, int dim,
                                    void* d_out, int out_dtype, int ldo, void* stream) {
    CMLB_REQUIRE(d_x && rows > 0 && dim > 0 && d_out && ldo >= dim && (!d_y || ldy >= dim), "cmlb200_residual_add: bad argument");
    CMLB_REQUIRE(!parts || (d_y && parts->top > 0 && parts->pos && parts->weight), "cmlb200_residual_add: parts without rows");
    return launch_residual(d_x, d_y, ldy, parts, d_w_post, nullptr, eps, rows, dim, nullptr, d_out, out_dtype, ldo, 1, as_stream(stream));
}

extern "C" int cmlb200_embed_streams(const void* d_table, int dtype, const int* d_tokens, float scale, int streams, int rows, int width, int vocab,
                                     float* d_x, void* stream) {
    CMLB_REQUIRE(d_table && d_tokens && d_x && streams > 0 && rows > 0 && width > 0 && vocab > 0, "cmlb200_embed_streams: bad argument");
    CMLB_REQUIRE(dtype == CMLB200_DT_F32 || dtype == CMLB200_DT_BF16, "cmlb200_embed_streams: dtype %d", dtype);
    const bool vec = width % 4 == 0 && (((uintptr_t)d_table | (uintptr_t)d_x) & 15) == 0;
    const dim3 grid(rows, rows < 64 ? (width + 1023) / 1024 : 1);
#define ES_LAUNCH(T, W) CMLB_CUDA(launch_chain(embed_streams_kernel<T, W>, grid, dim3(256), 0, 1, as_stream(stream), (const T*)d_table, d_tokens, scale, streams, width, vocab, d_x))
    if (dtype == CMLB200_DT_BF16) { if (vec) ES_LAUNCH(__nv_bfloat16, 4); else ES_LAUNCH(__nv_bfloat16, 1); }
    else { if (vec) ES_LAUNCH(float, 4); else ES_LAUNCH(float, 1); }
#undef ES_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_stream_join(const cmlb200_streams* hc, float* d_x, const float* d_y, int ldy, const cmlb200_join* j, const float* d_w_next, float eps,
                                   int rows, int width, const int* d_row_idx, void* d_out, int out_dtype, int ldo, void* stream) {
    CMLB_REQUIRE(hc && d_x && rows > 0 && width > 0 && (d_y || d_w_next), "cmlb200_stream_join: bad argument");
    CMLB_REQUIRE(hc->streams > 0 && hc->streams <= 8 && (!d_y || (hc->mix && hc->out)), "cmlb200_stream_join: %d streams", hc->streams);
    CMLB_REQUIRE(!d_w_next || (d_out && ldo >= width), "cmlb200_stream_join: no output for the normed rows");
    CMLB_REQUIRE(!(d_y && d_row_idx) && (!d_y || ldy >= width) && (!j || d_y), "cmlb200_stream_join: a row list goes with the norm-only form");
    CMLB_REQUIRE(out_dtype == CMLB200_DT_F32 || out_dtype == CMLB200_DT_BF16, "cmlb200_stream_join: dtype %d", out_dtype);
    const cmlb200_moe* parts = j ? j->parts : nullptr;
    const bool self = parts && parts->identity > 0;
    CMLB_REQUIRE(!parts || (parts->top > 0 && parts->pos && parts->weight), "cmlb200_stream_join: parts without rows");
    CMLB_REQUIRE(!self || (j->h && parts->self && ldo >= width), "cmlb200_stream_join: identity experts without their rows");
    CMLB_REQUIRE(!j || !j->add || j->ld_add >= width, "cmlb200_stream_join: stride %d", j->ld_add);
    const size_t smem = (size_t)((width + 3) / 4) * 16;
    CMLB_REQUIRE(smem <= 200 * 1024, "cmlb200_stream_join: rows of %d elements do not fit shared memory", width);
    const void *h = self ? j->h : nullptr, *add = j ? j->add : nullptr;
    const int ld_add = j ? j->ld_add : 0;
    const bool vec = width % 4 == 0 && (!d_y || ldy % 4 == 0) && (!d_w_next || ldo % 4 == 0) && ld_add % 4 == 0 &&
                     (((uintptr_t)d_x | (uintptr_t)d_y | (uintptr_t)d_w_next | (uintptr_t)d_out | (uintptr_t)add) & 15) == 0;
    int threads = 256;
    if (rows <= 2 * cmlb_num_sms()) while (threads < 1024 && threads * 4 < width) threads *= 2;
    if (hc->streams > 2 && threads > 512) threads = 512;               // registers
    static size_t attr[12][kMaxDevices] = {};
#define SJ_LAUNCH(TO, S, W, slot)                                                                                                        do {                                                                                                                                    auto kern = stream_join_kernel<TO, S, W>;                                                                                           CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                                CMLB_CUDA(launch_chain(kern, dim3(rows), dim3(threads), smem, 1, as_stream(stream), *hc, d_x, d_y, ldy, parts ? parts->top : 0,                                (const int*)(parts ? parts->pos : nullptr), (const float*)(parts ? parts->weight : nullptr),                                         (const float*)(self ? parts->self : nullptr), (const TO*)h, (const float*)add, ld_add, d_w_next, eps, width, d_row_idx,                                (TO*)d_out, ldo));                                                                                       } while (0)
#define SJ_WIDTH(TO, S, slot) do { if (vec) SJ_LAUNCH(TO, S, 4, slot); else SJ_LAUNCH(TO, S, 1, slot + 1); } while (0)
#define SJ_STREAMS(TO, slot) do { if (hc->streams <= 2) SJ_WIDTH(TO, 2, slot); else if (hc->streams <= 4) SJ_WIDTH(TO, 4, slot + 2); else SJ_WIDTH(TO, 8, slot + 4); } while (0)
    if (out_dtype == CMLB200_DT_BF16) SJ_STREAMS(__nv_bfloat16, 0);
    else SJ_STREAMS(float, 6);
#undef SJ_STREAMS
#undef SJ_WIDTH
#undef SJ_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_gated_join_rows(const cmlb200_gated_join* j, float* d_x, const float* d_w_next, float norm_eps, int rows, int width, void* d_out, int out_dtype, int ldo,
                                       void* stream) {
    static const char* who = "cmlb200_gated_join_rows";
    CMLB_REQUIRE(j && d_x && rows > 0 && width > 0 && j->a && j->ga && j->ldm >= width && j->ldg >= width, "%s: bad argument", who);
    CMLB_REQUIRE((!j->b || (j->a_norm && j->b_norm)) && (!j->f || (j->gf && j->ldf >= width)), "%s: norms or gates are missing", who);
    CMLB_REQUIRE(!j->parts || (j->f && j->parts->top > 0 && j->parts->identity == 0 && j->parts->pos && j->parts->weight), "%s: parts without rows", who);
    CMLB_REQUIRE(!j->table || (j->tokens && j->vocab > 0 && (j->table_dtype == CMLB200_DT_F32 || j->table_dtype == CMLB200_DT_BF16)), "%s: table without tokens", who);
    CMLB_REQUIRE((out_dtype == CMLB200_DT_F32 || out_dtype == CMLB200_DT_BF16) && (!d_w_next || (d_out && ldo >= width)), "%s: no output for the normed rows", who);
    const size_t smem = (size_t)((width + 3) / 4) * 16;
    CMLB_REQUIRE(smem <= 200 * 1024, "%s: rows of %d elements do not fit shared memory", who, width);
    const bool vec = width % 4 == 0 && j->ldm % 4 == 0 && j->ldg % 4 == 0 && (!j->f || j->ldf % 4 == 0) && (!d_w_next || ldo % 4 == 0) &&
                     (((uintptr_t)d_x | (uintptr_t)d_w_next | (uintptr_t)d_out | (uintptr_t)j->a | (uintptr_t)j->b | (uintptr_t)j->a_norm | (uintptr_t)j->b_norm | (uintptr_t)j->f |
                       (uintptr_t)j->ga | (uintptr_t)j->gf) & 15) == 0;
    int threads = 256;
    if (rows <= 2 * cmlb_num_sms()) while (threads < 1024 && threads * 4 < width) threads *= 2;
    const cmlb200_moe* parts = j->parts;
    static size_t attr[8][kMaxDevices] = {};
#define GJ_LAUNCH(TO, TE, W, slot)                                                                                                    \
    do {                                                                                                                              \
        auto kern = gated_join_kernel<TO, TE, W>;                                                                                     \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                          \
        CMLB_CUDA(launch_chain(kern, dim3(rows), dim3(threads), smem, 1, as_stream(stream), *j, parts ? parts->top : 0,               \
                               (const int*)(parts ? parts->pos : nullptr), (const float*)(parts ? parts->weight : nullptr), d_x, d_w_next, norm_eps, width, (TO*)d_out, ldo)); \
    } while (0)
#define GJ_WIDTH(TO, TE, slot) do { if (vec) GJ_LAUNCH(TO, TE, 4, slot); else GJ_LAUNCH(TO, TE, 1, slot + 1); } while (0)
#define GJ_TABLE(TO, slot) do { if (j->table && j->table_dtype == CMLB200_DT_F32) GJ_WIDTH(TO, float, slot); else GJ_WIDTH(TO, __nv_bfloat16, slot + 2); } while (0)
    if (out_dtype == CMLB200_DT_BF16) GJ_TABLE(__nv_bfloat16, 0);
    else GJ_TABLE(float, 4);
#undef GJ_TABLE
#undef GJ_WIDTH
#undef GJ_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_norm_columns(const float* d_x, int ld, int col, int n, const float* d_w, float eps, int rows, void* d_out, int out_dtype, int ldo, void* stream) {
    CMLB_REQUIRE(d_x && d_w && d_out && col >= 0 && n > 0 && rows > 0 && ld >= col + n && ldo >= n, "cmlb200_norm_columns: bad argument");
    CMLB_REQUIRE(out_dtype == CMLB200_DT_F32 || out_dtype == CMLB200_DT_BF16, "cmlb200_norm_columns: dtype %d", out_dtype);
#define NC_LAUNCH(TO) CMLB_CUDA(launch_chain(norm_columns_kernel<TO>, dim3(rows), dim3(256), 0, 1, as_stream(stream), d_x, ld, col, n, d_w, eps, (TO*)d_out, ldo))
    if (out_dtype == CMLB200_DT_BF16) NC_LAUNCH(__nv_bfloat16);
    else NC_LAUNCH(float);
#undef NC_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_act_rows_f32(const float* d_z, int ld, int rows, int ff, int act, float* d_f, int ldf, void* stream) {
    CMLB_REQUIRE(d_z && d_f && rows > 0 && ff > 0 && ld >= ff && ldf >= ff, "cmlb200_act_rows_f32: bad argument");
    CMLB_REQUIRE(act == CMLB200_ACT_SILU || act == CMLB200_ACT_GELU_TANH || act == CMLB200_ACT_GELU_ERF, "cmlb200_act_rows_f32: activation %d", act);
    CMLB_CUDA(launch_chain(act_rows_f32_kernel, dim3(rows, (ff + 1023) / 1024), dim3(256), 0, 1, as_stream(stream), d_z, ld, ff, act, d_f, ldf));
    return CMLB200_OK;
}

extern "C" int cmlb200_pack_columns(const float* d_x, int ld, int col, int n, int more, int at, int rows, uint16_t* d_out_bf16, int ldo, void* stream) {
    CMLB_REQUIRE(d_x && d_out_bf16 && col >= 0 && n > 0 && more >= 0 && rows > 0 && ld >= col + n + more && ldo >= n && (!more || (at >= n && ldo >= at + more)),
                 "cmlb200_pack_columns: bad argument");
    CMLB_CUDA(launch_chain(pack_columns_kernel, dim3(rows), dim3(256), 0, 1, as_stream(stream), d_x, ld, col, n, more, at, (__nv_bfloat16*)d_out_bf16, ldo));
    return CMLB200_OK;
}

extern "C" int cmlb200_poly_norm(const float* d_z, int ld, int rows, int ff, const float* d_coef, float eps, void* d_f, int out_dtype, int ldf, void* stream) {
    CMLB_REQUIRE(d_z && d_coef && d_f && rows > 0 && ff > 0 && ld >= ff && ldf >= ff, "cmlb200_poly_norm: bad argument");
    CMLB_REQUIRE(out_dtype == CMLB200_DT_F32 || out_dtype == CMLB200_DT_BF16, "cmlb200_poly_norm: dtype %d", out_dtype);
    const size_t smem = (size_t)((ff + 3) / 4) * 16;
    CMLB_REQUIRE(smem <= 200 * 1024, "cmlb200_poly_norm: rows of %d elements do not fit shared memory", ff);
    const bool vec = ff % 4 == 0 && ld % 4 == 0 && ldf % 4 == 0 && (((uintptr_t)d_z | (uintptr_t)d_f) & 15) == 0;
    int threads = 256;
    if (rows <= 2 * cmlb_num_sms()) while (threads < 1024 && threads * 4 < ff) threads *= 2;
    static size_t attr[4][kMaxDevices] = {};
#define PN_LAUNCH(TO, V, slot)                                                                                                      \
    do {                                                                                                                            \
        auto kern = poly_norm_kernel<TO, V>;                                                                                        \
        CMLB_CUDA(cmlb_ensure_smem(kern, smem, attr[slot]));                                                                        \
        CMLB_CUDA(launch_chain(kern, dim3(rows), dim3(threads), smem, 1, as_stream(stream), d_z, ld, ff, d_coef, eps, (TO*)d_f, ldf)); \
    } while (0)
    if (out_dtype == CMLB200_DT_BF16) { if (vec) PN_LAUNCH(__nv_bfloat16, true, 0); else PN_LAUNCH(__nv_bfloat16, false, 1); }
    else { if (vec) PN_LAUNCH(float, true, 2); else PN_LAUNCH(float, false, 3); }
#undef PN_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_qk_norm_append(const cmlb200_attn* a, float* d_qkv, int ld, const int* d_row_pos, const int* d_row_slot, int rows,
                                      void* stream) {
    CMLB_REQUIRE(a && d_qkv && d_row_pos && d_row_slot && rows > 0, "cmlb200_qk_norm_append: bad argument");
    const int rc = cmlb200_attn_check_(a, "cmlb200_qk_norm_append");
    if (rc) return rc;
    CMLB_REQUIRE(ld >= a->heads * a->dim + a->kv_heads * (a->dim + (a->keys_as_values ? 0 : a->vdim)), "cmlb200_qk_norm_append: row stride %d", ld);
    const size_t smem = a->head_norm ? (size_t)(a->heads + a->kv_heads) * 4 : 0;
    CMLB_REQUIRE(smem <= 40 * 1024, "cmlb200_qk_norm_append: %d heads", a->heads);
    cudaStream_t st = as_stream(stream);
    const bool vec = a->dim % 4 == 0 && a->vdim % 4 == 0 && ld % 4 == 0 && (((uintptr_t)d_qkv | (uintptr_t)a->q_norm | (uintptr_t)a->k_norm) & 15) == 0;
#define QK_LAUNCH(KV, V) CMLB_CUDA(launch_chain(qk_norm_append_kernel<KV, V>, dim3(rows), dim3(256), smem, 1, st, d_qkv, ld, d_row_pos, d_row_slot, *a, (KV*)a->k_pool, (KV*)a->v_pool))
    if (a->cache_dtype == CMLB200_DT_F32) { if (vec) QK_LAUNCH(float, true); else QK_LAUNCH(float, false); }
    else { if (vec) QK_LAUNCH(__half, true); else QK_LAUNCH(__half, false); }
#undef QK_LAUNCH
    return CMLB200_OK;
}

extern "C" int cmlb200_glu_rows_f32(const float* d_gu, int ld, int rows, int ff, int act, float* d_f, int ldf, void* stream) {
    CMLB_REQUIRE(d_gu && d_f && rows > 0 && ff > 0 && ldf >= ff && ld >= 2 * ((ff + 15) & ~15), "cmlb200_glu_rows_f32: bad argument");
    CMLB_CUDA(launch_chain(glu_rows_f32_kernel, dim3(rows, (ff + 1023) / 1024), dim3(256), 0, 1, as_stream(stream), d_gu, ld, ff, act, 0.f, d_f, ldf));
    return CMLB200_OK;
}

extern "C" int cmlb200_moe_glu_rows_f32(const float* d_gu, int ld, int rows, int ff, int act, float limit, float* d_f, int ldf, void* stream) {
    CMLB_REQUIRE(d_gu && d_f && rows > 0 && ff > 0 && ldf >= ff && ld >= 2 * ((ff + 15) & ~15), "cmlb200_moe_glu_rows_f32: bad argument");
    CMLB_CUDA(launch_chain(glu_rows_f32_kernel, dim3(rows, (ff + 1023) / 1024), dim3(256), 0, 1, as_stream(stream), d_gu, ld, ff, act, limit, d_f, ldf));
    return CMLB200_OK;
}

extern "C" int cmlb200_advance_tokens(const int* d_picked, int rows, int* d_tokens, int* d_pos, int* d_hist, int* d_step, void* stream) {
    CMLB_REQUIRE(d_picked && d_tokens && d_pos && d_hist && d_step && rows > 0, "cmlb200_advance_tokens: bad argument");
    CMLB_CUDA(launch_chain(advance_tokens_kernel, dim3(1), dim3(128), 0, 1, as_stream(stream), d_picked, rows, d_tokens, d_pos, d_hist, d_step));
    return CMLB200_OK;
}
