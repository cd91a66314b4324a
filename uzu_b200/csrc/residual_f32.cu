// Glue kernels of the parallel-block family (f32 residual stream): grouped RMS norm, norm (RMS, Dynamic Tanh or layer norm) with residual add and
// the next norm, a residual kept as several mixed streams with the next layer norm, embedding rows into f32, the token-gated gelu unit, the clamped gated unit, tanh, residual add, logit cap, and the routers (by table or by the largest logits: expert-sorted pair lists + weighted, optionally
// gated combine). Everything is f32 arithmetic.
#include "common.cuh"

namespace uzu {

// one CTA per (row, group); a thread keeps up to 8 of the part's elements in registers between the sum and the scaling
__global__ void __launch_bounds__(256) group_rms_norm_kernel(const uzu_group_rms_norm_args a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float red[32];
    const uint32_t row = blockIdx.x, g = blockIdx.y;
    const uint32_t src = a.row_indices ? reinterpret_cast<const uint32_t*>(a.row_indices)[row] : row;
    const uint32_t part = a.n / a.groups, base = g * part;
    const float* in = reinterpret_cast<const float*>(a.input) + (size_t)src * a.in_stride + base;
    float* out = reinterpret_cast<float*>(a.output) + (size_t)row * a.out_stride + base;
    const float* sc = a.scales ? reinterpret_cast<const float*>(a.scales) + base : nullptr;
    float* out2 = a.output2 ? reinterpret_cast<float*>(a.output2) + (size_t)row * a.out_stride + base : nullptr;
    const float* sc2 = a.scales2 ? reinterpret_cast<const float*>(a.scales2) + base : nullptr;
    constexpr int KEEP = 8;
    float v[KEEP];
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        v[j] = i < part ? in[i] : 0.0f;
    }
#pragma unroll
    for (int j = 0; j < KEEP; ++j) ss = fmaf(v[j], v[j], ss);
    for (uint32_t i = threadIdx.x + KEEP * blockDim.x; i < part; i += blockDim.x) ss = fmaf(in[i], in[i], ss);
    ss = block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)part + a.epsilon);
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        if (i < part) {
            out[i] = sc ? v[j] * inv * sc[i] : v[j] * inv;
            if (out2) out2[i] = sc2 ? v[j] * inv * sc2[i] : v[j] * inv;
        }
    }
    for (uint32_t i = threadIdx.x + KEEP * blockDim.x; i < part; i += blockDim.x) {
        out[i] = sc ? in[i] * inv * sc[i] : in[i] * inv;
        if (out2) out2[i] = sc2 ? in[i] * inv * sc2[i] : in[i] * inv;
    }
}

// One CTA per row. RMS norm: the row's sum of squares first; Dynamic Tanh is elementwise. With a residual the normed row is added into
// it (times mult) and the updated row can be normed again for the next sublayer; a second RMS norm takes a second sum over the row.
__device__ __forceinline__ float norm_add_value(uint32_t kind, float x, float mean, float inv, float alpha, const float* w, const float* b, uint32_t i) {
    float v = kind == 1 ? tanhf(alpha * x) : (x - mean) * inv;
    if (w) v *= w[i];
    if (b) v += b[i];
    return v;
}

// Dynamic Tanh in and (if any) out: nothing crosses an element, so the work is cut over elements, not rows.
__global__ void __launch_bounds__(256) norm_add_elementwise_kernel(const uzu_norm_add_args a) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t row = blockIdx.y, i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= a.n) return;
    const float* w = reinterpret_cast<const float*>(a.weight);
    const float* b = reinterpret_cast<const float*>(a.bias);
    const float v = norm_add_value(1, reinterpret_cast<const float*>(a.input)[(size_t)row * a.in_stride + i], 0.0f, 1.0f, a.alpha, w, b, i);
    float* out = a.output ? reinterpret_cast<float*>(a.output) + (size_t)row * a.n : nullptr;
    if (!a.residual) { out[i] = v; return; }
    float* res = reinterpret_cast<float*>(a.residual) + (size_t)row * a.n;
    const float x = fmaf(a.mult, v, res[i]);
    res[i] = x;
    if (out) out[i] = norm_add_value(1, x, 0.0f, 1.0f, a.next_alpha, reinterpret_cast<const float*>(a.next_weight), reinterpret_cast<const float*>(a.next_bias), i);
}

// One CTA per row; a thread keeps up to KEEP of the row's elements (input, weights, residual) in registers, all requested before the
// first sum, so a decode step's single row costs one round trip to memory and not one per pass over the row.
__global__ void __launch_bounds__(256) norm_add_kernel(const uzu_norm_add_args a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float red[32];
    const uint32_t row = blockIdx.x;
    const float* in = reinterpret_cast<const float*>(a.input) + (size_t)row * a.in_stride;
    const float* w = reinterpret_cast<const float*>(a.weight);
    const float* b = reinterpret_cast<const float*>(a.bias);
    const float* nw = reinterpret_cast<const float*>(a.next_weight);
    const float* nb = reinterpret_cast<const float*>(a.next_bias);
    float* res = a.residual ? reinterpret_cast<float*>(a.residual) + (size_t)row * a.n : nullptr;
    float* out = a.output ? reinterpret_cast<float*>(a.output) + (size_t)row * a.n : nullptr;
    constexpr int KEEP = 8;
    float x[KEEP], wv[KEEP], bv[KEEP], rv[KEEP], nwv[KEEP], nbv[KEEP];
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        const bool ok = i < a.n;
        x[j] = ok ? in[i] : 0.0f;
        wv[j] = (ok && w) ? w[i] : 1.0f;
        bv[j] = (ok && b) ? b[i] : 0.0f;
        rv[j] = (ok && res) ? res[i] : 0.0f;
        nwv[j] = (ok && nw) ? nw[i] : 1.0f;
        nbv[j] = (ok && nb) ? nb[i] : 0.0f;
    }
    float inv = 1.0f, mean = 0.0f;
    if (a.kind == 2) {
        float s = 0.0f;
#pragma unroll
        for (int j = 0; j < KEEP; ++j) s += x[j];
        for (uint32_t i = threadIdx.x + KEEP * blockDim.x; i < a.n; i += blockDim.x) s += in[i];
        mean = block_sum(s, red) / (float)a.n;
    }
    if (a.kind != 1) {
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < KEEP; ++j) {
            const float d = threadIdx.x + j * blockDim.x < a.n ? x[j] - mean : 0.0f;
            ss = fmaf(d, d, ss);
        }
        for (uint32_t i = threadIdx.x + KEEP * blockDim.x; i < a.n; i += blockDim.x) { const float d = in[i] - mean; ss = fmaf(d, d, ss); }
        ss = block_sum(ss, red);
        inv = 1.0f / sqrtf(ss / (float)a.n + a.epsilon);
    }
    // first norm, and the residual add
    __nv_bfloat16* copy = a.residual_bf16 ? reinterpret_cast<__nv_bfloat16*>(a.output) + (size_t)row * a.n : nullptr;
    float s2 = 0.0f, ss2 = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        float v = (a.kind == 1 ? tanhf(a.alpha * x[j]) : (x[j] - mean) * inv) * wv[j] + bv[j];
        if (res) v = fmaf(a.mult, v, rv[j]);
        x[j] = v;
        if (i < a.n) {
            ss2 = fmaf(v, v, ss2);
            s2 += v;
            if (res) res[i] = v;
            else out[i] = v;
            if (copy) copy[i] = __float2bfloat16_rn(v);
        }
    }
    for (uint32_t i = threadIdx.x + KEEP * blockDim.x; i < a.n; i += blockDim.x) {
        float v = norm_add_value(a.kind, in[i], mean, inv, a.alpha, w, b, i);
        if (res) { v = fmaf(a.mult, v, res[i]); res[i] = v; }          // read back below by the thread that wrote it
        else out[i] = v;
        if (copy) copy[i] = __float2bfloat16_rn(v);
        ss2 = fmaf(v, v, ss2);
        s2 += v;
    }
    if (!res || !out || copy) return;
    float inv2 = 1.0f, mean2 = 0.0f;
    if (a.next_kind == 2) {         // the deviations need the mean: a second sum over the row
        mean2 = block_sum(s2, red) / (float)a.n;
        ss2 = 0.0f;
#pragma unroll
        for (int j = 0; j < KEEP; ++j) {
            const float d = threadIdx.x + j * blockDim.x < a.n ? x[j] - mean2 : 0.0f;
            ss2 = fmaf(d, d, ss2);
        }
        for (uint32_t i = threadIdx.x + KEEP * blockDim.x; i < a.n; i += blockDim.x) { const float d = res[i] - mean2; ss2 = fmaf(d, d, ss2); }
    }
    if (a.next_kind != 1) {
        ss2 = block_sum(ss2, red);
        inv2 = 1.0f / sqrtf(ss2 / (float)a.n + a.epsilon);
    }
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        if (i < a.n) out[i] = (a.next_kind == 1 ? tanhf(a.next_alpha * x[j]) : (x[j] - mean2) * inv2) * nwv[j] + nbv[j];
    }
    for (uint32_t i = threadIdx.x + KEEP * blockDim.x; i < a.n; i += blockDim.x) out[i] = norm_add_value(a.next_kind, res[i], mean2, inv2, a.next_alpha, nw, nb, i);
}

// The same for RMS and layer norms without a second norm over rows of whole float4 that a CTA holds in registers (n <= 8 * threads): 16-byte
// requests, all of a thread's in flight at once.
__global__ void __launch_bounds__(512) norm_add_vec_kernel(const uzu_norm_add_args a) {
    pdl_launch_dependents();
    __shared__ float red[32];
    constexpr int KEEP = 2;
    const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f), one = make_float4(1.0f, 1.0f, 1.0f, 1.0f);
    const uint32_t row = blockIdx.x, n4 = a.n / 4;
    float4 x[KEEP], w[KEEP], b[KEEP], r[KEEP];
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        w[j] = (a.weight && i < n4) ? reinterpret_cast<const float4*>(a.weight)[i] : one;
        b[j] = (a.bias && i < n4) ? reinterpret_cast<const float4*>(a.bias)[i] : zero;
    }
    pdl_wait();
    const float4* in = reinterpret_cast<const float4*>(reinterpret_cast<const float*>(a.input) + (size_t)row * a.in_stride);
    float4* res = a.residual ? reinterpret_cast<float4*>(a.residual) + (size_t)row * n4 : nullptr;
    float s = 0.0f, ss = 0.0f, mean = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        x[j] = i < n4 ? in[i] : zero;
        r[j] = (res && i < n4) ? res[i] : zero;
        s += (x[j].x + x[j].y) + (x[j].z + x[j].w);
    }
    if (a.kind == 2) mean = block_sum(s, red) / (float)a.n;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        if (threadIdx.x + j * blockDim.x < n4) {
            x[j].x -= mean; x[j].y -= mean; x[j].z -= mean; x[j].w -= mean;
            ss += (x[j].x * x[j].x + x[j].y * x[j].y) + (x[j].z * x[j].z + x[j].w * x[j].w);
        }
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)a.n + a.epsilon);
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        if (i >= n4) continue;
        float4 v = make_float4(x[j].x * inv * w[j].x + b[j].x, x[j].y * inv * w[j].y + b[j].y, x[j].z * inv * w[j].z + b[j].z, x[j].w * inv * w[j].w + b[j].w);
        if (!res) {
            reinterpret_cast<float4*>(a.output)[(size_t)row * n4 + i] = v;
            continue;
        }
        v = make_float4(fmaf(a.mult, v.x, r[j].x), fmaf(a.mult, v.y, r[j].y), fmaf(a.mult, v.z, r[j].z), fmaf(a.mult, v.w, r[j].w));
        res[i] = v;
        if (a.residual_bf16) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
            reinterpret_cast<uint2*>(a.output)[(size_t)row * n4 + i] = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        }
    }
}

// One CTA per row of a residual kept as several streams: begin from the embedding, or take a sublayer's result in; then the next reader's
// weighted sum of the streams and its layer norm. A thread keeps up to KEEP elements of that sum in registers between the passes over it.
template <int MAXS>
__global__ void __launch_bounds__(MAXS > 4 ? 256 : 1024) stream_mix_kernel(const uzu_stream_mix_args a) {
    pdl_launch_dependents();
    __shared__ float red[32], cmix[MAXS * MAXS], cout[MAXS], cread[MAXS];
    const uint32_t row = blockIdx.x, S = a.streams;
    for (uint32_t i = threadIdx.x; i < MAXS * MAXS; i += blockDim.x) {          // coefficients (weights: not written by the launch before)
        const uint32_t s = i / MAXS, t = i % MAXS;
        cmix[i] = (a.y && s < S && t < S) ? reinterpret_cast<const float*>(a.mix)[s * S + t] : 0.0f;
        if (i < MAXS) {
            cout[i] = (a.y && i < S) ? reinterpret_cast<const float*>(a.out)[i] : 0.0f;
            cread[i] = i < S ? (a.read ? reinterpret_cast<const float*>(a.read)[i] : 1.0f) : 0.0f;
        }
    }
    pdl_wait();
    __syncthreads();
    float* x = reinterpret_cast<float*>(a.x) + (size_t)row * S * a.n;
    const float* y = a.y ? reinterpret_cast<const float*>(a.y) + (size_t)row * a.n : nullptr;
    float* u_out = a.u ? reinterpret_cast<float*>(a.u) + (size_t)row * a.n : nullptr;
    const uint32_t tok = a.token_ids ? reinterpret_cast<const uint32_t*>(a.token_ids)[row] : 0u;
    auto element = [&](uint32_t i) {
        float xs[MAXS], u = 0.0f;
        if (a.token_ids) {
            float e = 0.0f;
            if (tok < a.vocab) {
                const size_t at = (size_t)tok * a.n + i;
                e = a.table_dt == UZU_DT_F32 ? reinterpret_cast<const float*>(a.table)[at] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(a.table)[at]);
            }
#pragma unroll
            for (int s = 0; s < MAXS; ++s) xs[s] = e;
        } else {
#pragma unroll
            for (int s = 0; s < MAXS; ++s) xs[s] = (uint32_t)s < S ? x[(size_t)s * a.n + i] : 0.0f;
        }
        const float yy = y ? y[i] : 0.0f;
#pragma unroll
        for (int t = 0; t < MAXS; ++t) {
            if ((uint32_t)t < S) {
                float v = xs[t];
                if (y) {
                    v = cout[t] * yy;
#pragma unroll
                    for (int s = 0; s < MAXS; ++s) v = fmaf(cmix[s * MAXS + t], xs[s], v);
                }
                if (y || a.token_ids) x[(size_t)t * a.n + i] = v;
                u = fmaf(cread[t], v, u);
            }
        }
        if (u_out) u_out[i] = u;
        return u;
    };
    auto again = [&](uint32_t i) {          // the same sum from the streams this thread has just stored (or that nobody changed)
        float u = 0.0f;
        for (uint32_t t = 0; t < S; ++t) u = fmaf(cread[t], x[(size_t)t * a.n + i], u);
        return u;
    };
    constexpr int KEEP = 8;
    float u[KEEP], sum = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        u[j] = i < a.n ? element(i) : 0.0f;
        sum += u[j];
    }
    for (uint32_t i = threadIdx.x + KEEP * blockDim.x; i < a.n; i += blockDim.x) sum += element(i);
    if (!a.output) return;
    const float mean = block_sum(sum, red) / (float)a.n;
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const float d = threadIdx.x + j * blockDim.x < a.n ? u[j] - mean : 0.0f;
        ss = fmaf(d, d, ss);
    }
    for (uint32_t i = threadIdx.x + KEEP * blockDim.x; i < a.n; i += blockDim.x) { const float d = again(i) - mean; ss = fmaf(d, d, ss); }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)a.n + a.epsilon);
    const float* w = reinterpret_cast<const float*>(a.weight);
    auto store = [&](uint32_t i, float v) {
        v = (v - mean) * inv * w[i];
        if (a.output_bf16) reinterpret_cast<__nv_bfloat16*>(a.output)[(size_t)row * a.n + i] = __float2bfloat16_rn(v);
        else reinterpret_cast<float*>(a.output)[(size_t)row * a.n + i] = v;
    };
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        if (i < a.n) store(i, u[j]);
    }
    for (uint32_t i = threadIdx.x + KEEP * blockDim.x; i < a.n; i += blockDim.x) store(i, again(i));
}

// The same for rows of whole float4 that a CTA holds in registers (n <= 8 * threads): 16-byte requests, all of a thread's in flight at once.
template <int MAXS>
__global__ void __launch_bounds__(512) stream_mix_vec_kernel(const uzu_stream_mix_args a) {
    pdl_launch_dependents();
    __shared__ float red[32], cmix[MAXS * MAXS], cout[MAXS], cread[MAXS];
    const uint32_t row = blockIdx.x, S = a.streams, n4 = a.n / 4;
    if (threadIdx.x < MAXS * MAXS) {
        const uint32_t s = threadIdx.x / MAXS, t = threadIdx.x % MAXS;
        cmix[threadIdx.x] = (a.y && s < S && t < S) ? reinterpret_cast<const float*>(a.mix)[s * S + t] : 0.0f;
        if (s == 0) {
            cout[t] = (a.y && t < S) ? reinterpret_cast<const float*>(a.out)[t] : 0.0f;
            cread[t] = t < S ? (a.read ? reinterpret_cast<const float*>(a.read)[t] : 1.0f) : 0.0f;
        }
    }
    constexpr int KEEP = 2;
    const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    float4 w[KEEP];
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        w[j] = (a.output && i < n4) ? reinterpret_cast<const float4*>(a.weight)[i] : zero;
    }
    pdl_wait();
    float4* x = reinterpret_cast<float4*>(a.x) + (size_t)row * S * n4;
    const float4* y = a.y ? reinterpret_cast<const float4*>(a.y) + (size_t)row * n4 : nullptr;
    float4 xs[KEEP][MAXS], yy[KEEP], u[KEEP];
    if (a.token_ids) {
        const uint32_t tok = reinterpret_cast<const uint32_t*>(a.token_ids)[row];
#pragma unroll
        for (int j = 0; j < KEEP; ++j) {
            const uint32_t i = threadIdx.x + j * blockDim.x;
            float4 e = zero;
            if (tok < a.vocab && i < n4) {
                const size_t at = (size_t)tok * n4 + i;
                if (a.table_dt == UZU_DT_F32) {
                    e = reinterpret_cast<const float4*>(a.table)[at];
                } else {
                    const uint2 b = reinterpret_cast<const uint2*>(a.table)[at];
                    e = make_float4(__uint_as_float(b.x << 16), __uint_as_float(b.x & 0xffff0000u), __uint_as_float(b.y << 16), __uint_as_float(b.y & 0xffff0000u));
                }
            }
#pragma unroll
            for (int s = 0; s < MAXS; ++s) xs[j][s] = e;
            yy[j] = zero;
        }
    } else {
#pragma unroll
        for (int j = 0; j < KEEP; ++j) {
            const uint32_t i = threadIdx.x + j * blockDim.x;
#pragma unroll
            for (int s = 0; s < MAXS; ++s) xs[j][s] = ((uint32_t)s < S && i < n4) ? x[(size_t)s * n4 + i] : zero;
            yy[j] = (y && i < n4) ? y[i] : zero;
        }
    }
    __syncthreads();
    float sum = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        u[j] = zero;
#pragma unroll
        for (int t = 0; t < MAXS; ++t) {
            if ((uint32_t)t < S) {
                float4 v = xs[j][t];
                if (y) {
                    const float co = cout[t];
                    v = make_float4(co * yy[j].x, co * yy[j].y, co * yy[j].z, co * yy[j].w);
#pragma unroll
                    for (int s = 0; s < MAXS; ++s) {
                        const float m = cmix[s * MAXS + t];
                        v.x = fmaf(m, xs[j][s].x, v.x); v.y = fmaf(m, xs[j][s].y, v.y); v.z = fmaf(m, xs[j][s].z, v.z); v.w = fmaf(m, xs[j][s].w, v.w);
                    }
                }
                if ((y || a.token_ids) && i < n4) x[(size_t)t * n4 + i] = v;
                const float cr = cread[t];
                u[j].x = fmaf(cr, v.x, u[j].x); u[j].y = fmaf(cr, v.y, u[j].y); u[j].z = fmaf(cr, v.z, u[j].z); u[j].w = fmaf(cr, v.w, u[j].w);
            }
        }
        if (a.u && i < n4) reinterpret_cast<float4*>(a.u)[(size_t)row * n4 + i] = u[j];
        sum += (u[j].x + u[j].y) + (u[j].z + u[j].w);              // (zero past the row)
    }
    if (!a.output) return;
    const float mean = block_sum(sum, red) / (float)a.n;
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        if (threadIdx.x + j * blockDim.x < n4) {
            u[j].x -= mean; u[j].y -= mean; u[j].z -= mean; u[j].w -= mean;
            ss += (u[j].x * u[j].x + u[j].y * u[j].y) + (u[j].z * u[j].z + u[j].w * u[j].w);
        }
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)a.n + a.epsilon);
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const uint32_t i = threadIdx.x + j * blockDim.x;
        if (i >= n4) continue;
        const float4 v = make_float4(u[j].x * inv * w[j].x, u[j].y * inv * w[j].y, u[j].z * inv * w[j].z, u[j].w * inv * w[j].w);
        if (a.output_bf16) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
            reinterpret_cast<uint2*>(a.output)[(size_t)row * n4 + i] = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        } else {
            reinterpret_cast<float4*>(a.output)[(size_t)row * n4 + i] = v;
        }
    }
}

template <typename TW>
__global__ void token_gate_kernel(const uzu_token_gate_args a) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (size_t)a.rows * a.n) return;
    const uint32_t r = (uint32_t)(idx / a.n), i = (uint32_t)(idx % a.n);
    const uint32_t tok = reinterpret_cast<const uint32_t*>(a.token_ids)[r];
    float e = 0.0f;
    if (tok < a.vocab) {
        const TW* t = reinterpret_cast<const TW*>(a.table) + (size_t)tok * a.table_stride + a.column + i;
        if constexpr (sizeof(TW) == 2) e = __bfloat162float(*t);
        else e = *t;
    }
    const float z = reinterpret_cast<const float*>(a.z)[idx];
    const float g = 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
    reinterpret_cast<float*>(a.out)[idx] = g * e;
}

// a thread per channel pair (2i, 2i + 1): the two share the angle of a sinusoidal position vector
template <typename TW>
__global__ void embedding_f32_kernel(const uzu_embedding_f32_args a) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t row = blockIdx.y, i = blockIdx.x * blockDim.x + threadIdx.x, c0 = 2 * i, n = a.n;
    const uint32_t tok = reinterpret_cast<const uint32_t*>(a.token_ids)[row];
    if (c0 >= n) return;
    const bool two = c0 + 1 < n;
    float v[2] = {0.0f, 0.0f};
    if (tok < a.vocab) {
        const TW* t = reinterpret_cast<const TW*>(a.table) + (size_t)tok * n + c0;
        if constexpr (sizeof(TW) == 2) { v[0] = __bfloat162float(t[0]); if (two) v[1] = __bfloat162float(t[1]); }
        else { v[0] = t[0]; if (two) v[1] = t[1]; }
    }
    v[0] *= a.scale; v[1] *= a.scale;
    if (a.position_turns) {
        const uint32_t p = (a.dynamic_position ? *reinterpret_cast<const uint32_t*>(a.dynamic_position) : a.prefix) + row;
        const double turns = (double)p * reinterpret_cast<const double*>(a.position_turns)[i];
        float s, c;
        sincospif(2.0f * (float)(turns - rint(turns)), &s, &c);
        v[0] += s; v[1] += c;
    }
    float* out = reinterpret_cast<float*>(a.output) + (size_t)row * n + c0;
    out[0] = v[0];
    if (two) out[1] = v[1];
    if (a.rows_bf16) {
        __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(a.rows_bf16) + (size_t)row * n + c0;
        o[0] = __float2bfloat16_rn(v[0]);
        if (two) o[1] = __float2bfloat16_rn(v[1]);
    }
}

__device__ __forceinline__ float glu_value(uint32_t kind, float g, float u, float limit, float alpha) {
    if (kind == 0) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit) + 1.0f;
        return g * (1.0f / (1.0f + expf(-alpha * g))) * u;
    }
    if (kind == 1) return g * (1.0f / (1.0f + expf(-g))) * u;
    return 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
}

// VEC elements of one row per thread (f a multiple of VEC, 16-byte aligned operands when VEC = 4)
template <int VEC>
__global__ void __launch_bounds__(256) glu_kernel(const uzu_glu_args a) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t idx = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (idx >= (size_t)a.rows * a.f) return;
    const uint32_t r = (uint32_t)(idx / a.f), c = (uint32_t)(idx % a.f);
    const float* src = reinterpret_cast<const float*>(a.gate_up) + (size_t)r * 2 * a.f + c;
    const float limit = (a.group_offsets && r >= reinterpret_cast<const uint32_t*>(a.group_offsets)[a.last_group]) ? a.limit_last : a.limit;
    float v[VEC];
    if constexpr (VEC == 4) {
        const float4 g = *reinterpret_cast<const float4*>(src), u = *reinterpret_cast<const float4*>(src + a.f);
        v[0] = glu_value(a.kind, g.x, u.x, limit, a.alpha); v[1] = glu_value(a.kind, g.y, u.y, limit, a.alpha);
        v[2] = glu_value(a.kind, g.z, u.z, limit, a.alpha); v[3] = glu_value(a.kind, g.w, u.w, limit, a.alpha);
        if (a.output_bf16) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
            *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(a.output) + idx) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        } else {
            *reinterpret_cast<float4*>(reinterpret_cast<float*>(a.output) + idx) = make_float4(v[0], v[1], v[2], v[3]);
        }
    } else {
        v[0] = glu_value(a.kind, src[0], src[a.f], limit, a.alpha);
        if (a.output_bf16) reinterpret_cast<__nv_bfloat16*>(a.output)[idx] = __float2bfloat16_rn(v[0]);
        else reinterpret_cast<float*>(a.output)[idx] = v[0];
    }
}

__global__ void rows_to_bf16_kernel(const float* src, uint32_t src_stride, __nv_bfloat16* dst, uint32_t rows, uint32_t n) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (size_t)rows * n) return;
    const size_t r = idx / n, c = idx % n;
    dst[idx] = __float2bfloat16_rn(src[r * src_stride + c]);
}

__global__ void unary_f32_kernel(const float* in, uint32_t in_stride, float* out, uint32_t out_stride, uint32_t rows, uint32_t n, uint32_t op) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (size_t)rows * n) return;
    const size_t r = idx / n, c = idx % n;
    const float v = in[r * in_stride + c];
    out[r * out_stride + c] = op == 0 ? tanhf(v) : v;
}

__global__ void residual_add_kernel(float* x, const float* a, const float* b, uint32_t length) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= length) return;
    float s = a[idx];
    if (b) s += b[idx];
    x[idx] += s;
}

__global__ void logit_cap_f32_kernel(float* logits, __nv_bfloat16* copy, uint32_t length, float cap, uint32_t has_cap) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= length) return;
    float v = logits[idx];
    if (has_cap) {
        v = cap * tanhf(v / cap);
        logits[idx] = v;
    }
    if (copy) copy[idx] = __float2bfloat16_rn(v);
}

// Counting sort of the (row, slot) pairs by expert, by one CTA: `pe` (shared memory) holds the expert of every pair, `counts`
// (shared memory, [experts + 1]) is scratch. Pairs of one expert keep token order, so the lists do not depend on the thread schedule.
__device__ void route_sort_pairs(const uint16_t* pe, uint32_t* counts, uint32_t pairs, uint32_t top, uint32_t experts, uint32_t* offsets,
                                 uint32_t* rows_map, uint32_t* pair_pos) {
    for (uint32_t e = threadIdx.x; e <= experts; e += blockDim.x) counts[e] = 0;
    __syncthreads();
    for (uint32_t base = 0; base < pairs; base += blockDim.x) {      // one shared-memory add per (warp, expert): lanes with the same expert elect a leader
        const uint32_t p = base + threadIdx.x;
        const bool valid = p < pairs;
        const uint32_t e = valid ? pe[p] : 0x10000u + (threadIdx.x & 31);
        const uint32_t same = __match_any_sync(0xffffffffu, e);
        if (valid && (threadIdx.x & 31) == (uint32_t)(__ffs(same) - 1)) atomicAdd(&counts[e + 1], (uint32_t)__popc(same));
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        for (uint32_t e = 0; e < experts; ++e) counts[e + 1] += counts[e];
    }
    __syncthreads();
    for (uint32_t e = threadIdx.x; e <= experts; e += blockDim.x) offsets[e] = counts[e];
    __syncthreads();
    // Stable placement, counts[e] now being the next free position of expert e: pairs are taken in chunks of one per thread, the warps of
    // a chunk one after the other; within a warp the lanes that hold the same expert are ranked by lane and their leader moves the cursor.
    const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    // Few experts: every warp of a chunk counts its pairs per expert at once, one thread per expert turns the counts into the warps' start
    // positions (in warp order), then every pair is placed: four barriers per chunk instead of one per warp.
    constexpr uint32_t kFew = 64;
    __shared__ uint32_t warp_start[32][kFew];
    if (experts <= kFew && warps <= 32 && pairs > 32) {        // (a single warp's worth of pairs takes the loop below in one step)
        for (uint32_t base = 0; base < pairs; base += blockDim.x) {
            for (uint32_t i = threadIdx.x; i < 32 * kFew; i += blockDim.x) (&warp_start[0][0])[i] = 0;
            __syncthreads();
            const uint32_t p = base + threadIdx.x;
            const bool valid = p < pairs;
            const uint32_t e = valid ? pe[p] : 0x10000u + lane;
            const uint32_t same = __match_any_sync(0xffffffffu, e);
            const uint32_t rank = __popc(same & ((1u << lane) - 1u));
            if (valid && rank == 0) warp_start[warp][e] = __popc(same);
            __syncthreads();
            if (threadIdx.x < experts) {
                uint32_t cur = counts[threadIdx.x];
                for (uint32_t w = 0; w < warps; ++w) {
                    const uint32_t c = warp_start[w][threadIdx.x];
                    warp_start[w][threadIdx.x] = cur;
                    cur += c;
                }
                counts[threadIdx.x] = cur;
            }
            __syncthreads();
            if (valid) {
                const uint32_t at = warp_start[warp][e] + rank;
                rows_map[at] = p / top;
                pair_pos[p] = at;
            }
            __syncthreads();
        }
        return;
    }
    for (uint32_t base = 0; base < pairs; base += blockDim.x) {
        const uint32_t p = base + threadIdx.x;
        const bool valid = p < pairs;
        const uint32_t e = valid ? pe[p] : 0x10000u + lane;          // idle lanes match nobody
        const uint32_t busy = min(warps, (pairs - base + 31) / 32);
        for (uint32_t w = 0; w < busy; ++w) {
            if (warp == w) {
                const uint32_t same = __match_any_sync(0xffffffffu, e);
                const uint32_t rank = __popc(same & ((1u << lane) - 1u));
                uint32_t at = 0;
                if (valid && rank == 0) {
                    at = counts[e];
                    counts[e] = at + __popc(same);
                }
                at = __shfl_sync(0xffffffffu, at, __ffs(same) - 1);
                if (valid) {
                    rows_map[at + rank] = p / top;
                    pair_pos[p] = at + rank;
                }
            }
            __syncthreads();
        }
    }
}

// One CTA; rows * top <= 1024 * top pairs; experts <= 8192. The experts of a token come from a table row.
__global__ void __launch_bounds__(1024) table_route_kernel(const uzu_table_route_args a) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ uint32_t counts[];   // [experts + 1]
    const uint32_t* tokens = reinterpret_cast<const uint32_t*>(a.token_ids);
    const int32_t* table = reinterpret_cast<const int32_t*>(a.table);
    const uint32_t pairs = a.rows * a.top;
    uint16_t* pe = reinterpret_cast<uint16_t*>(counts + a.experts + 1);   // expert of every pair, staged once
    for (uint32_t p = threadIdx.x; p < pairs; p += blockDim.x) {
        const uint32_t tok = tokens[p / a.top];
        const int32_t e = tok < a.vocab ? table[(size_t)tok * a.top + p % a.top] : 0;
        pe[p] = (uint16_t)((e >= 0 && (uint32_t)e < a.experts) ? (uint32_t)e : 0u);
    }
    __syncthreads();
    route_sort_pairs(pe, counts, pairs, a.top, a.experts, reinterpret_cast<uint32_t*>(a.group_offsets), reinterpret_cast<uint32_t*>(a.rows_map),
                     reinterpret_cast<uint32_t*>(a.pair_pos));
}

// One CTA, a warp per row: `top` rounds, each picking the best (logit, lower index first) that comes after the previous pick in that
// order, so no list of the picked experts is kept. Weights: exp(z - z_first) over the sum of the picked ones, or (weight_kind 1) the
// sigmoid of every picked logit on its own, or (weight_kind 2) the sigmoids of the picked ones over their sum, picked by sigmoid + correction
// among the experts of the best groups. compact_weight gets the same weights in the expert-sorted order of the pair list.
// MODE 0: choice and pair lists in one CTA (short passes). Long passes with a scratch: MODE 1 makes the choice over many CTAs (a warp per
// row, the picked experts go to the scratch), MODE 2 is the one CTA that sorts them into the pair lists.
constexpr int ROUTE_GROUPS = 8;      // words of 32 groups
constexpr size_t ROUTE_SMEM = 192 * 1024;   // the experts' counters and the pairs of a pass

template <int MODE>
__global__ void __launch_bounds__(MODE == 1 ? 256 : 1024) topk_route_kernel(const uzu_topk_route_args a) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ uint32_t counts[];   // [experts + 1]
    const uint32_t slots = a.top + a.always, experts = a.experts + a.always, pairs = a.rows * slots;      // with the experts that every row uses
    uint16_t* pe_shared = reinterpret_cast<uint16_t*>(counts + experts + 1);
    uint16_t* pe = MODE == 1 ? reinterpret_cast<uint16_t*>(a.scratch) : pe_shared;
    const float* bias = reinterpret_cast<const float*>(a.bias);
    float* weight = reinterpret_cast<float*>(a.pair_weight);
    const uint32_t lane = threadIdx.x & 31, warp = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), warps = gridDim.x * (blockDim.x >> 5);
    if constexpr (MODE == 2) {
        const uint16_t* chosen = reinterpret_cast<const uint16_t*>(a.scratch);
        for (uint32_t p = threadIdx.x; p < pairs; p += blockDim.x) pe_shared[p] = chosen[p];
    } else {
    // a lane keeps the logit of expert `lane` of its row in a register for all rounds, and requests the next row's before it works on this one
    auto first_logit = [&](uint32_t r) {
        return (r < a.rows && lane < a.experts) ? reinterpret_cast<const float*>(a.logits)[(size_t)r * a.logits_stride + lane] + (bias ? bias[lane] : 0.0f) : 0.0f;
    };
    const bool corrected = a.weight_kind == 2;
    const float* correction = reinterpret_cast<const float*>(a.correction);
    const uint32_t groups = corrected && a.choice_groups > 1 ? a.choice_groups : 1u, group_size = a.experts / groups;
    const float own_correction = corrected && correction && lane < a.experts ? correction[lane] : 0.0f;
    // what the choice goes by: the logit, or its sigmoid plus the expert's correction
    auto score_of = [&](float z, uint32_t e) {
        return corrected ? 1.0f / (1.0f + expf(-z)) + (e == lane ? own_correction : correction ? correction[e] : 0.0f) : z;
    };
    float next_z = first_logit(warp);
    for (uint32_t r = warp; r < a.rows; r += warps) {
        const float* z = reinterpret_cast<const float*>(a.logits) + (size_t)r * a.logits_stride;
        const float own_z = score_of(next_z, lane);
        next_z = first_logit(r + warps);
        // lane g % 32 holds group g's score and whether its experts can be chosen (at most 32 * GROUPS groups)
        float group_score[ROUTE_GROUPS];
        uint32_t open_groups = 0xFFFFFFFFu;                  // bit g / 32 of lane g % 32
        if (groups > 1) {
#pragma unroll
            for (int q = 0; q < ROUTE_GROUPS; ++q) group_score[q] = -INFINITY;
            for (uint32_t g = 0; g < groups; ++g) {          // the two largest choice scores of the group, over the warp
                float hi = -INFINITY, lo = -INFINITY;
                for (uint32_t e0 = g * group_size; e0 < (g + 1) * group_size; e0 += 32) {
                    // lane l looks at the expert of this batch that it also owns in the rounds below (e % 32 == l), so own_z serves batch 0
                    const uint32_t base = e0 & ~31u, e = base + lane + (base + lane < e0 ? 32u : 0u);
                    if (e < (g + 1) * group_size && e < e0 + 32) {
                        const float v = e == lane ? own_z : score_of(z[e] + (bias ? bias[e] : 0.0f), e);
                        if (v > hi) { lo = hi; hi = v; }
                        else if (v > lo) lo = v;
                    }
                }
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) {
                    const float oh = __shfl_xor_sync(0xffffffffu, hi, o), ol = __shfl_xor_sync(0xffffffffu, lo, o);
                    lo = fmaxf(fminf(hi, oh), fmaxf(lo, ol));
                    hi = fmaxf(hi, oh);
                }
                if (group_size == 1) lo = 0.0f;
#pragma unroll
                for (int q = 0; q < ROUTE_GROUPS; ++q)
                    if (g == 32u * q + lane) group_score[q] = hi + lo;
            }
            open_groups = 0;
            for (uint32_t k = 0; k < a.choice_keep; ++k) {   // the best group that is not open yet, the lower index first
                float best = -INFINITY;
                uint32_t at = 0xFFFFFFFFu;
#pragma unroll
                for (int q = 0; q < ROUTE_GROUPS; ++q) {
                    const uint32_t g = 32u * q + lane;
                    if (g < groups && !(open_groups >> q & 1u) && (at == 0xFFFFFFFFu || group_score[q] > best)) { best = group_score[q]; at = g; }
                }
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) {
                    const float ov = __shfl_xor_sync(0xffffffffu, best, o);
                    const uint32_t oi = __shfl_xor_sync(0xffffffffu, at, o);
                    if (oi != 0xFFFFFFFFu && (at == 0xFFFFFFFFu || ov > best || (ov == best && oi < at))) { best = ov; at = oi; }
                }
                if (at != 0xFFFFFFFFu && (at & 31u) == lane) open_groups |= 1u << (at >> 5);
            }
        }
        float prev_v = INFINITY, first = 0.0f, sum = 0.0f;
        uint32_t prev_i = 0;
        bool any = false;
        for (uint32_t s = 0; s < a.top; ++s) {
            float best_v = -INFINITY;
            uint32_t best_i = 0xFFFFFFFFu;
            for (uint32_t e0 = 0; e0 < a.experts; e0 += 32) {
                const uint32_t e = e0 + lane, g = groups > 1 ? min(e, a.experts - 1) / group_size : 0u;
                const uint32_t open = __shfl_sync(0xffffffffu, open_groups, g & 31u);
                if (e >= a.experts || !(open >> (g >> 5) & 1u)) continue;
                const float v = e == lane ? own_z : score_of(z[e] + (bias ? bias[e] : 0.0f), e);
                const bool after = !any || v < prev_v || (v == prev_v && e > prev_i);
                if (after && (best_i == 0xFFFFFFFFu || v > best_v)) { best_v = v; best_i = e; }    // ascending e: the first of equals stays
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ov = __shfl_xor_sync(0xffffffffu, best_v, o);
                const uint32_t oi = __shfl_xor_sync(0xffffffffu, best_i, o);
                if (oi != 0xFFFFFFFFu && (best_i == 0xFFFFFFFFu || ov > best_v || (ov == best_v && oi < best_i))) { best_v = ov; best_i = oi; }
            }
            if (best_i == 0xFFFFFFFFu) { best_i = 0; best_v = first; }      // fewer usable logits than slots (NaNs): keep the lists well-formed
            if (!any) first = best_v;
            any = true;
            prev_v = best_v; prev_i = best_i;
            const float w = corrected ? 1.0f / (1.0f + expf(-(z[best_i] + (bias ? bias[best_i] : 0.0f))))
                                      : a.weight_kind == 1 ? 1.0f / (1.0f + expf(-best_v)) : expf(best_v - first);
            sum += w;
            if (lane == 0) {
                pe[r * slots + s] = (uint16_t)best_i;
                weight[r * slots + s] = w;
            }
        }
        __syncwarp();
        if (lane < a.top && a.weight_kind != 1) {
            for (uint32_t s = lane; s < a.top; s += 32) {
                const float w = weight[r * slots + s];
                weight[r * slots + s] = corrected ? w / (sum + 1e-20f) * a.weight_scale : w / sum;
            }
        }
        for (uint32_t s = lane; s < a.always; s += 32) {
            pe[r * slots + a.top + s] = (uint16_t)(a.experts + s);
            weight[r * slots + a.top + s] = 1.0f;
        }
    }
    }
    if constexpr (MODE == 1) return;
    __syncthreads();
    route_sort_pairs(pe_shared, counts, pairs, slots, experts, reinterpret_cast<uint32_t*>(a.group_offsets), reinterpret_cast<uint32_t*>(a.rows_map),
                     reinterpret_cast<uint32_t*>(a.pair_pos));
    if (a.compact_weight) {
        __syncthreads();
        const uint32_t* pos = reinterpret_cast<const uint32_t*>(a.pair_pos);
        float* cw = reinterpret_cast<float*>(a.compact_weight);
        for (uint32_t p = threadIdx.x; p < pairs; p += blockDim.x) cw[pos[p]] = weight[p];
    }
}

__global__ void routed_combine_kernel(const uzu_routed_combine_args a) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (size_t)a.rows * a.n) return;
    const size_t r = idx / a.n, c = idx % a.n;
    const float* pairs = reinterpret_cast<const float*>(a.pairs);
    const uint32_t* pair_pos = reinterpret_cast<const uint32_t*>(a.pair_pos);
    const float* pw = reinterpret_cast<const float*>(a.pair_weight);
    float s = 0.0f;
    for (uint32_t k = 0; k < a.top; ++k) {
        const float v = pairs[(size_t)pair_pos[r * a.top + k] * a.n + c];
        s = pw ? fmaf(pw[r * a.top + k], v, s) : s + v;
    }
    s *= a.weight;
    if (a.gate) {
        float g = reinterpret_cast<const float*>(a.gate)[r * a.gate_ld + c];
        if (a.gate_bias) g += reinterpret_cast<const float*>(a.gate_bias)[c];
        s *= 1.0f / (1.0f + expf(-g));
    }
    if (a.col_scale) s *= reinterpret_cast<const float*>(a.col_scale)[c];
    float* out = reinterpret_cast<float*>(a.output);
    out[idx] = a.accumulate ? out[idx] + s : s;
}

static inline unsigned blocks256(size_t n) { return (unsigned)((n + 255) / 256); }

}  // namespace uzu

extern "C" {
using namespace uzu;

void uzu_group_rms_norm_encode(uzu_command_buffer* cmd, const uzu_group_rms_norm_args* a) {
    if (!encodable(cmd, "group_rms_norm")) return;
    if (!a->input || !a->output || a->groups == 0 || a->n % a->groups != 0) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, "group_rms_norm: null operand or the row is not divisible into the groups");
        return;
    }
    if (a->rows == 0 || a->n == 0) return;
    uzu_group_rms_norm_args b = *a;
    if (!b.in_stride) b.in_stride = b.n;
    if (!b.out_stride) b.out_stride = b.n;
    launch(cmd, "group_rms_norm_kernel", group_rms_norm_kernel, dim3(b.rows, b.groups), dim3(256), 0, b);
}

void uzu_embedding_f32_scaled_encode(uzu_command_buffer* cmd, uint64_t token_ids, uint64_t table, uint32_t weights_dt, uint64_t output, uint32_t rows,
                                     uint32_t vocab, uint32_t n, float scale) {
    uzu_embedding_f32_args a{};
    a.token_ids = token_ids; a.table = table; a.output = output; a.rows = rows; a.vocab = vocab; a.n = n; a.weights_dt = weights_dt; a.scale = scale;
    uzu_embedding_f32_position_encode(cmd, &a);
}

void uzu_embedding_f32_position_encode(uzu_command_buffer* cmd, const uzu_embedding_f32_args* a) {
    if (!encodable(cmd, "embedding_f32") || a->rows == 0 || a->n == 0) return;
    if (!a->token_ids || !a->table || !a->output || (a->weights_dt != UZU_DT_BF16 && a->weights_dt != UZU_DT_F32)) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, "embedding_f32: null operand or bad table type");
        return;
    }
    const dim3 grid(blocks256((a->n + 1) / 2), a->rows);
    if (a->weights_dt == UZU_DT_BF16) launch(cmd, "embedding_f32_kernel", embedding_f32_kernel<__nv_bfloat16>, grid, dim3(256), 0, *a);
    else launch(cmd, "embedding_f32_kernel", embedding_f32_kernel<float>, grid, dim3(256), 0, *a);
}

void uzu_glu_encode(uzu_command_buffer* cmd, const uzu_glu_args* a) {
    if (!encodable(cmd, "glu")) return;
    if (!a->gate_up || !a->output || a->kind > 2) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, "glu: null operand or unknown unit");
        return;
    }
    if (a->rows == 0 || a->f == 0) return;
    const size_t n = (size_t)a->rows * a->f;
    if (a->f % 4 == 0 && (a->gate_up & 15) == 0 && (a->output & 15) == 0) launch(cmd, "glu_kernel", glu_kernel<4>, dim3(blocks256(n / 4)), dim3(256), 0, *a);
    else launch(cmd, "glu_kernel", glu_kernel<1>, dim3(blocks256(n)), dim3(256), 0, *a);
}

void uzu_embedding_f32_encode(uzu_command_buffer* cmd, uint64_t token_ids, uint64_t table, uint32_t weights_dt, uint64_t output, uint32_t rows,
                              uint32_t vocab, uint32_t n) {
    uzu_embedding_f32_scaled_encode(cmd, token_ids, table, weights_dt, output, rows, vocab, n, 1.0f);
}

void uzu_norm_add_encode(uzu_command_buffer* cmd, const uzu_norm_add_args* a) {
    if (!encodable(cmd, "norm_add")) return;
    if (!a->input || (!a->residual && !a->output) || a->kind > 2 || a->next_kind > 2 || (a->residual_bf16 && (!a->residual || !a->output))) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, "norm_add: null operand or unknown norm kind");
        return;
    }
    if (a->rows == 0 || a->n == 0) return;
    uzu_norm_add_args b = *a;
    if (!b.in_stride) b.in_stride = b.n;
    if (b.kind == 1 && !b.residual_bf16 && (!b.residual || !b.output || b.next_kind == 1))
        launch(cmd, "norm_add_elementwise_kernel", norm_add_elementwise_kernel, dim3((b.n + 255) / 256, b.rows), dim3(256), 0, b);
    else if (b.kind != 1 && (!b.residual || !b.output || b.residual_bf16) && b.n % 4 == 0 && b.n <= 4096 && b.in_stride % 4 == 0 &&
             ((b.input | b.weight | b.bias | b.residual | b.output) & 15) == 0)
        launch(cmd, "norm_add_kernel", norm_add_vec_kernel, dim3(b.rows), dim3(b.n <= 1024 ? 128 : b.n <= 2048 ? 256 : 512), 0, b);
    else
        launch(cmd, "norm_add_kernel", norm_add_kernel, dim3(b.rows), dim3(256), 0, b);
}

void uzu_stream_mix_encode(uzu_command_buffer* cmd, const uzu_stream_mix_args* a) {
    if (!encodable(cmd, "stream_mix")) return;
    if (!a->x || a->streams == 0 || a->streams > 16 || (a->y && (!a->mix || !a->out)) || (a->output && !a->weight) || (a->token_ids && (!a->table || a->y)) ||
        (a->token_ids && a->table_dt != UZU_DT_BF16 && a->table_dt != UZU_DT_F32)) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, "stream_mix: null operand, more than 16 streams, or a beginning that also takes a result in");
        return;
    }
    if (a->rows == 0 || a->n == 0) return;
    // rows of whole float4 up to 4096 elements, all row blocks 16-byte aligned
    const uint64_t blocks = a->x | a->y | a->u | a->weight | a->output | a->table;
    if (a->n % 4 == 0 && a->n <= 4096 && a->streams <= 4 && (blocks & 15) == 0) {
        const uint32_t t = a->n <= 1024 ? 128 : (a->n <= 2048 ? 256 : 512);
        if (a->streams <= 2) launch(cmd, "stream_mix_kernel", stream_mix_vec_kernel<2>, dim3(a->rows), dim3(t), 0, *a);
        else launch(cmd, "stream_mix_kernel", stream_mix_vec_kernel<4>, dim3(a->rows), dim3(t), 0, *a);
        return;
    }
    const uint32_t threads = (a->n <= 2048 || a->streams > 4) ? 256 : (a->n <= 4096 ? 512 : 1024);
    auto go = [&](auto kernel) { launch(cmd, "stream_mix_kernel", kernel, dim3(a->rows), dim3(threads), 0, *a); };
    if (a->streams <= 2) go(stream_mix_kernel<2>);
    else if (a->streams <= 4) go(stream_mix_kernel<4>);
    else go(stream_mix_kernel<16>);
}

void uzu_rows_to_bf16_encode(uzu_command_buffer* cmd, uint64_t src, uint32_t src_stride, uint64_t dst, uint32_t rows, uint32_t n) {
    if (!encodable(cmd, "rows_to_bf16") || rows == 0 || n == 0) return;
    if (!src || !dst || src_stride < n) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, "rows_to_bf16: null operand or a row stride below the row size");
        return;
    }
    launch(cmd, "rows_to_bf16_kernel", rows_to_bf16_kernel, dim3(blocks256((size_t)rows * n)), dim3(256), 0, (const float*)src, src_stride, (__nv_bfloat16*)dst, rows, n);
}

void uzu_token_gate_encode(uzu_command_buffer* cmd, const uzu_token_gate_args* a) {
    if (!encodable(cmd, "token_gate")) return;
    if (!a->z || !a->token_ids || !a->table || !a->out || (a->weights_dt != UZU_DT_BF16 && a->weights_dt != UZU_DT_F32) || a->column + a->n > a->table_stride) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, "token_gate: null operand, bad table type, or columns outside the table");
        return;
    }
    if (a->rows == 0 || a->n == 0) return;
    const dim3 grid(blocks256((size_t)a->rows * a->n));
    if (a->weights_dt == UZU_DT_BF16) launch(cmd, "token_gate_kernel", token_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, *a);
    else launch(cmd, "token_gate_kernel", token_gate_kernel<float>, grid, dim3(256), 0, *a);
}

void uzu_clamped_glu_encode(uzu_command_buffer* cmd, uint64_t gate_up, uint64_t output, uint32_t rows, uint32_t f, float limit, float alpha) {
    uzu_glu_args a{};
    a.gate_up = gate_up; a.output = output; a.rows = rows; a.f = f; a.kind = 0; a.limit = limit; a.alpha = alpha;
    uzu_glu_encode(cmd, &a);
}

void uzu_silu_glu_encode(uzu_command_buffer* cmd, uint64_t gate_up, uint64_t output, uint32_t rows, uint32_t f) {
    uzu_glu_args a{};
    a.gate_up = gate_up; a.output = output; a.rows = rows; a.f = f; a.kind = 1;
    uzu_glu_encode(cmd, &a);
}

void uzu_unary_f32_encode(uzu_command_buffer* cmd, uint64_t input, uint32_t in_stride, uint64_t output, uint32_t out_stride, uint32_t rows,
                          uint32_t n, uint32_t op) {
    if (!encodable(cmd, "unary_f32") || rows == 0 || n == 0) return;
    launch(cmd, "unary_f32_kernel", unary_f32_kernel, dim3(blocks256((size_t)rows * n)), dim3(256), 0, (const float*)input, in_stride, (float*)output, out_stride, rows, n, op);
}

void uzu_residual_add_encode(uzu_command_buffer* cmd, uint64_t x, uint64_t a, uint64_t b, uint32_t length) {
    if (!encodable(cmd, "residual_add") || length == 0) return;
    launch(cmd, "residual_add_kernel", residual_add_kernel, dim3(blocks256(length)), dim3(256), 0, (float*)x, (const float*)a, (const float*)b, length);
}

void uzu_logit_cap_f32_encode(uzu_command_buffer* cmd, uint64_t logits_f32, uint64_t logits_bf16, uint32_t length, float cap, uint32_t has_cap) {
    if (!encodable(cmd, "logit_cap_f32") || length == 0) return;
    launch(cmd, "logit_cap_f32_kernel", logit_cap_f32_kernel, dim3(blocks256(length)), dim3(256), 0, (float*)logits_f32, (__nv_bfloat16*)logits_bf16, length, cap, has_cap);
}

void uzu_table_route_encode(uzu_command_buffer* cmd, const uzu_table_route_args* a) {
    if (!encodable(cmd, "table_route")) return;
    if (!a->token_ids || !a->table || !a->group_offsets || !a->rows_map || !a->pair_pos || a->top == 0 || a->experts == 0 || a->experts > 8192) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, "table_route: null operand or bad expert count");
        return;
    }
    if (a->rows == 0) return;
    const size_t smem = (a->experts + 1) * sizeof(uint32_t) + (size_t)a->rows * a->top * sizeof(uint16_t);
    if (smem > 48 * 1024) {
        cmd->record_error(UZU_ERROR_UNSUPPORTED, "table_route: rows * top too large for one pass");
        return;
    }
    launch(cmd, "table_route_kernel", table_route_kernel, dim3(1), dim3(1024), smem, *a);
}

void uzu_topk_route_encode(uzu_command_buffer* cmd, const uzu_topk_route_args* a) {
    if (!encodable(cmd, "topk_route")) return;
    if (!a->logits || !a->group_offsets || !a->rows_map || !a->pair_pos || !a->pair_weight || a->top == 0 || a->experts == 0 || a->experts > 8192 ||
        a->top > a->experts || a->logits_stride < a->experts || a->weight_kind > 2 || (a->always && a->weight_kind != 2)) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, "topk_route: null operand or bad expert / top count");
        return;
    }
    if (a->weight_kind == 2 && a->choice_groups > 1 &&
        (a->choice_groups > 32 * ROUTE_GROUPS || a->experts % a->choice_groups || a->choice_keep == 0 || a->choice_keep > a->choice_groups ||
         a->top > a->experts / a->choice_groups * a->choice_keep)) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, "topk_route: the groups must divide the experts (at most 256 groups), and the kept ones hold at least `top` experts");
        return;
    }
    if (a->rows == 0) return;
    const size_t smem = (a->experts + a->always + 1) * sizeof(uint32_t) + (size_t)a->rows * (a->top + a->always) * sizeof(uint16_t);
    if (smem > ROUTE_SMEM) {
        cmd->record_error(UZU_ERROR_UNSUPPORTED, "topk_route: rows * top too large for one pass");
        return;
    }
    static std::atomic<uint64_t> done[2];
    if (a->scratch && a->rows >= 64) {          // the choice over many CTAs (8 rows each), then the one CTA that builds the lists
        opt_in_dynamic_smem(cmd, topk_route_kernel<2>, (int)ROUTE_SMEM, done[1]);
        launch(cmd, "topk_route_kernel", topk_route_kernel<1>, dim3((a->rows + 7) / 8), dim3(256), 0, *a);
        launch(cmd, "topk_route_kernel", topk_route_kernel<2>, dim3(1), dim3(1024), smem, *a);
        return;
    }
    opt_in_dynamic_smem(cmd, topk_route_kernel<0>, (int)ROUTE_SMEM, done[0]);
    const uint32_t warps = std::min(32u, std::max(2u, a->rows));        // few rows: a small CTA, its barriers meet sooner
    launch(cmd, "topk_route_kernel", topk_route_kernel<0>, dim3(1), dim3(32 * warps), smem, *a);
}

void uzu_routed_combine_gated_encode(uzu_command_buffer* cmd, const uzu_routed_combine_args* a) {
    if (!encodable(cmd, "routed_combine") || a->rows == 0 || a->n == 0) return;
    if (!a->pairs || !a->pair_pos || !a->output || a->top == 0 || (a->gate_bias && !a->gate)) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, "routed_combine: null operand, or a gate bias without a gate");
        return;
    }
    uzu_routed_combine_args b = *a;
    if (!b.gate_ld) b.gate_ld = b.n;
    launch(cmd, "routed_combine_kernel", routed_combine_kernel, dim3(blocks256((size_t)b.rows * b.n)), dim3(256), 0, b);
}

void uzu_routed_combine_encode(uzu_command_buffer* cmd, uint64_t pairs, uint64_t pair_pos, uint64_t output, uint32_t rows, uint32_t top, uint32_t n,
                               float weight, uint32_t accumulate) {
    uzu_routed_combine_args a{};
    a.pairs = pairs; a.pair_pos = pair_pos; a.output = output; a.rows = rows; a.top = top; a.n = n; a.weight = weight; a.accumulate = accumulate;
    uzu_routed_combine_gated_encode(cmd, &a);
}

}  // extern "C"
