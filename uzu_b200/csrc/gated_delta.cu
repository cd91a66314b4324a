// Gated delta rule with one decay per head, for any head sizes, f32 throughout. Per head a state S [dim, vdim]:
//     S <- g S;  S <- S + k (beta (v - S^T k))^T;  o = S^T q
// with q, k, v behind a short causal convolution per channel and silu, q and k unit vectors, g = exp(-exp(A) softplus(.)), beta = sigmoid(.).
//
// A column of S (one value channel) needs no other column: S^T k and S^T q are dot products along it. So L neighbouring lanes own a column --
// lane part p holds the key channels {4 (i L + p) .. + 3}, NV float4 in registers -- and a token costs two dot products, two shuffle
// reductions over L lanes and no barrier at all. q and k rows are read from shared memory as float4 with the L parts side by side (128
// contiguous bytes at L = 8: no bank conflict, the columns of a warp share the read).
//   gated_delta_kernel       the tokens of a pass in order, 4 warps per CTA, grid (column blocks, heads). The prepared q / k / v / decay / beta
//                            rows arrive by cp.async one batch ahead. An element's arithmetic does not depend on how a prompt is cut.
//   delta_prepare_kernel     convolution, silu, unit vectors and gates of all tokens of a pass at once, a warp per (a few tokens, head).
//   gated_delta_step_kernel  one token with everything between the projections in one launch: a cluster of CL CTAs per head, each CTA owning
//                            vdim / CL columns; the state is requested before the previous kernel's results are waited for; the head's sum
//                            of squares meets through distributed shared memory in rank order; norm weight and silu gate applied on the way out.
// The convolution's earlier inputs live in a ring of `taps` rows indexed by position % taps: the step kernel writes the slot of its own token
// while all CTAs read the other taps - 1 slots, so no ordering between the CTAs is needed (several value heads may share a key head).
#include <type_traits>

#include "common.cuh"

namespace uzu {

namespace {

constexpr float kUnitEps = 1e-6f;

__device__ __forceinline__ float gd_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float gd_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float gd_decay(float a_log, float a) {
    const float softplus = fmaxf(a, 0.0f) + log1pf(expf(-fabsf(a)));
    return expf(-expf(a_log) * softplus);
}

__device__ __forceinline__ uint32_t gd_prefix(const uzu_delta_prepare_args& a) {
    return a.dynamic_position ? *reinterpret_cast<const uint32_t*>(a.dynamic_position) : a.prefix;
}

// silu of the convolution of channel c at row t of the pass (position prefix + t)
__device__ __forceinline__ float gd_conv(const uzu_delta_prepare_args& a, uint32_t channels, uint32_t prefix, uint32_t t, uint32_t c) {
    const float* proj = reinterpret_cast<const float*>(a.proj) + c;
    const float* w = reinterpret_cast<const float*>(a.conv) + (size_t)c * a.taps;
    const float* ring = reinterpret_cast<const float*>(a.ring) + c;
    float y = 0.0f;
    for (uint32_t j = 0; j < a.taps; ++j) {
        const uint32_t back = a.taps - 1 - j;                    // tokens before the current one
        float x = 0.0f;
        if (back <= t) x = proj[(size_t)(t - back) * a.stride];
        else if (back <= prefix + t) x = ring[(size_t)((prefix + t - back) % a.taps) * channels];
        y = fmaf(w[j], x, y);
    }
    return gd_silu(y);
}

// the convolution of channel c at position `prefix` without its last tap (all inputs come from the ring), and that tap's weight
__device__ __forceinline__ void gd_conv_past(const uzu_delta_prepare_args& a, uint32_t channels, uint32_t prefix, uint32_t c, float& past, float& tap) {
    const float* w = reinterpret_cast<const float*>(a.conv) + (size_t)c * a.taps;
    const float* ring = reinterpret_cast<const float*>(a.ring) + c;
    past = 0.0f;
    for (uint32_t j = 0; j + 1 < a.taps; ++j) {
        const uint32_t back = a.taps - 1 - j;
        if (back <= prefix) past = fmaf(w[j], ring[(size_t)((prefix - back) % a.taps) * channels], past);
    }
    tap = w[a.taps - 1];
}

__device__ __forceinline__ void gd_cp_async16(void* smem_ptr, const void* gmem_ptr) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem_ptr)), "l"(gmem_ptr) : "memory");
}
__device__ __forceinline__ void gd_cp_async4(void* smem_ptr, const void* gmem_ptr) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(smem_ptr)), "l"(gmem_ptr) : "memory");
}

template <int L>
__device__ __forceinline__ float gd_lane_sum(float v) {
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// v[0] of lane part p <- the sum over the L lanes of a column of v[p / (L / U)]  (U values, U <= L, both powers of two)
template <int U, int L>
__device__ __forceinline__ void gd_transpose_sum(float (&v)[U], uint32_t part) {
    int n = U;
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) {
        if (n > 1) {
            n >>= 1;
            const bool up = (part & o) != 0;
#pragma unroll
            for (int i = 0; i < U / 2; ++i) {
                if (i < n) {
                    const float keep = up ? v[i + n] : v[i], send = up ? v[i] : v[i + n];
                    v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                }
            }
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
        }
    }
}

template <int NV>
__device__ __forceinline__ float gd_dot(const float4 (&a)[NV], const float4 (&b)[NV]) {
    float x = 0.0f, y = 0.0f, z = 0.0f, w = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        x = fmaf(a[i].x, b[i].x, x);
        y = fmaf(a[i].y, b[i].y, y);
        z = fmaf(a[i].z, b[i].z, z);
        w = fmaf(a[i].w, b[i].w, w);
    }
    return (x + y) + (z + w);
}

// S <- g S + k u on a lane's channels
template <int NV>
__device__ __forceinline__ void gd_update(float4 (&s)[NV], const float4 (&k)[NV], float g, float u) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        s[i].x = fmaf(k[i].x, u, g * s[i].x);
        s[i].y = fmaf(k[i].y, u, g * s[i].y);
        s[i].z = fmaf(k[i].z, u, g * s[i].z);
        s[i].w = fmaf(k[i].w, u, g * s[i].w);
    }
}

}  // namespace

// A warp per (block of GP_ROWS tokens, unit): units [0, kv_heads) queries, [kv_heads, 2 kv_heads) keys, then the value heads, then one unit for
// the gates. NC = channels of a head per lane; the convolution's window of a channel slides through registers, so an input is read once.
constexpr int GP_ROWS = 8;

template <int TAPS, int NC>
__global__ void __launch_bounds__(128) delta_prepare_window_kernel(const uzu_delta_prepare_args a) {
    pdl_launch_dependents();
    const uint32_t lane = threadIdx.x & 31;
    const uint32_t units = 2 * a.kv_heads + a.heads + 1, blocks = (a.rows + GP_ROWS - 1) / GP_ROWS;
    const uint32_t item = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= blocks * units) return;
    const uint32_t t0 = item / units * GP_ROWS, unit = item % units, nr = min((uint32_t)GP_ROWS, a.rows - t0);
    const uint32_t kd = a.kv_heads * a.dim, channels = 2 * kd + a.heads * a.vdim, dim4 = (a.dim + 3) & ~3u;
    if (unit == units - 1) {
        pdl_wait();
        for (uint32_t i = lane; i < nr * a.heads; i += 32) {
            const uint32_t t = t0 + i / a.heads, h = i % a.heads;
            const float* row = reinterpret_cast<const float*>(a.proj) + (size_t)t * a.stride;
            reinterpret_cast<float*>(a.decay)[(size_t)t * a.heads + h] =
                gd_decay(reinterpret_cast<const float*>(a.a_log)[h], row[a.a_offset + h] + reinterpret_cast<const float*>(a.dt_bias)[h]);
            reinterpret_cast<float*>(a.beta)[(size_t)t * a.heads + h] = gd_sigmoid(row[a.b_offset + h]);
        }
        return;
    }
    const bool is_q = unit < a.kv_heads, is_v = unit >= 2 * a.kv_heads;
    const uint32_t head = is_q ? unit : (is_v ? unit - 2 * a.kv_heads : unit - a.kv_heads), n = is_v ? a.vdim : a.dim;
    const uint32_t c0 = is_q ? head * a.dim : (is_v ? 2 * kd + head * a.vdim : kd + head * a.dim);
    const uint32_t pad = is_v ? n : dim4;                        // q / k rows are padded to whole float4
    float* out = reinterpret_cast<float*>(is_q ? a.q : (is_v ? a.v : a.k)) + ((size_t)t0 * (is_v ? a.heads : a.kv_heads) + head) * pad;
    const size_t out_stride = (size_t)(is_v ? a.heads : a.kv_heads) * pad;
    const float* proj = reinterpret_cast<const float*>(a.proj) + (size_t)t0 * a.stride + c0;
    float w[NC][TAPS], x[NC][TAPS + GP_ROWS - 1];
#pragma unroll
    for (int i = 0; i < NC; ++i) {
        const uint32_t c = lane + 32u * i;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[i][j] = c < n ? reinterpret_cast<const float*>(a.conv)[(size_t)(c0 + c) * TAPS + j] : 0.0f;
    }
    pdl_wait();
    const uint32_t prefix = gd_prefix(a);
#pragma unroll
    for (int i = 0; i < NC; ++i) {
        const uint32_t c = lane + 32u * i;
#pragma unroll
        for (int j = 0; j < TAPS + GP_ROWS - 1; ++j) {
            const int t = j - (TAPS - 1);                        // row relative to the block's first
            float v = 0.0f;
            if (c < n) {
                if (t >= 0 || (uint32_t)(-t) <= t0) { if (t < (int)nr) v = proj[(ptrdiff_t)t * a.stride + c]; }
                else if ((uint32_t)(-t) <= prefix + t0)
                    v = reinterpret_cast<const float*>(a.ring)[(size_t)((prefix + t0 + t) % TAPS) * channels + c0 + c];
            }
            x[i][j] = v;
        }
    }
#pragma unroll
    for (int r = 0; r < GP_ROWS; ++r) {
        if ((uint32_t)r >= nr) break;
        float y[NC], f = 1.0f;
#pragma unroll
        for (int i = 0; i < NC; ++i) {
            float s = 0.0f;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) s = fmaf(w[i][j], x[i][r + j], s);
            y[i] = gd_silu(s);
        }
        if (!is_v) {
            float ss = 0.0f;
#pragma unroll
            for (int i = 0; i < NC; ++i) ss = fmaf(y[i], y[i], ss);      // (channels past the head hold zero)
            f = 1.0f / sqrtf(warp_sum(ss) + kUnitEps);
            if (is_q) f *= 1.0f / sqrtf((float)a.dim);
        }
#pragma unroll
        for (int i = 0; i < NC; ++i) {
            const uint32_t c = lane + 32u * i;
            if (c < pad) out[(size_t)r * out_stride + c] = y[i] * f;
        }
    }
}

// the same for any number of taps and any head size: a warp per (token, unit), every input read once per tap
__global__ void __launch_bounds__(128) delta_prepare_kernel(const uzu_delta_prepare_args a) {
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t lane = threadIdx.x & 31;
    const uint32_t units = 2 * a.kv_heads + a.heads + 1;
    const uint32_t item = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= a.rows * units) return;
    const uint32_t t = item / units, unit = item % units;
    const uint32_t kd = a.kv_heads * a.dim, channels = 2 * kd + a.heads * a.vdim, dim4 = (a.dim + 3) & ~3u;
    const uint32_t prefix = gd_prefix(a);
    if (unit < 2 * a.kv_heads) {
        const bool is_q = unit < a.kv_heads;
        const uint32_t head = is_q ? unit : unit - a.kv_heads;
        const uint32_t c0 = (is_q ? 0u : kd) + head * a.dim;
        float* out = reinterpret_cast<float*>(is_q ? a.q : a.k) + ((size_t)t * a.kv_heads + head) * dim4;
        constexpr int KEEP = 8;
        float x[KEEP], ss = 0.0f;
#pragma unroll
        for (int i = 0; i < KEEP; ++i) {
            const uint32_t c = lane + 32u * i;
            x[i] = c < a.dim ? gd_conv(a, channels, prefix, t, c0 + c) : 0.0f;
            ss = fmaf(x[i], x[i], ss);
        }
        for (uint32_t c = lane + 32u * KEEP; c < a.dim; c += 32) {          // long heads: the rest waits in the output row
            const float y = gd_conv(a, channels, prefix, t, c0 + c);
            out[c] = y;
            ss = fmaf(y, y, ss);
        }
        float f = 1.0f / sqrtf(warp_sum(ss) + kUnitEps);
        if (is_q) f *= 1.0f / sqrtf((float)a.dim);
#pragma unroll
        for (int i = 0; i < KEEP; ++i) {
            const uint32_t c = lane + 32u * i;
            if (c < dim4) out[c] = x[i] * f;                               // the pad channels hold zero
        }
        for (uint32_t c = lane + 32u * KEEP; c < dim4; c += 32) out[c] = c < a.dim ? out[c] * f : 0.0f;
    } else if (unit < 2 * a.kv_heads + a.heads) {
        const uint32_t h = unit - 2 * a.kv_heads;
        float* out = reinterpret_cast<float*>(a.v) + ((size_t)t * a.heads + h) * a.vdim;
        for (uint32_t c = lane; c < a.vdim; c += 32) out[c] = gd_conv(a, channels, prefix, t, 2 * kd + h * a.vdim + c);
    } else {
        const float* row = reinterpret_cast<const float*>(a.proj) + (size_t)t * a.stride;
        for (uint32_t h = lane; h < a.heads; h += 32) {
            reinterpret_cast<float*>(a.decay)[(size_t)t * a.heads + h] =
                gd_decay(reinterpret_cast<const float*>(a.a_log)[h], row[a.a_offset + h] + reinterpret_cast<const float*>(a.dt_bias)[h]);
            reinterpret_cast<float*>(a.beta)[(size_t)t * a.heads + h] = gd_sigmoid(row[a.b_offset + h]);
        }
    }
}

constexpr int GD_WARPS = 4;

template <int L, int NV>
constexpr int gd_batch() { return L * NV * 4 <= 256 ? 16 : (L * NV * 4 <= 512 ? 8 : 4); }

template <int L, int NV>
__global__ void __launch_bounds__(GD_WARPS * 32) gated_delta_kernel(const uzu_gated_delta_args ga) {
    constexpr int ROWF = L * NV * 4, BATCH = gd_batch<L, NV>(), CC = GD_WARPS * (32 / L), U = BATCH < 8 ? BATCH : 8;
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float gd_smem[];
    float* qs = gd_smem;                             // [2][BATCH][ROWF]
    float* ks = qs + 2 * BATCH * ROWF;               // [2][BATCH][ROWF]
    float* vs = ks + 2 * BATCH * ROWF;               // [2][BATCH][CC]
    float* gs = vs + 2 * BATCH * CC;                 // [2][BATCH] decay
    float* bs = gs + 2 * BATCH;                      // [2][BATCH] beta
    const uzu_delta_prepare_args& a = ga.prep;
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, part = lane % L;
    const uint32_t h = blockIdx.y, kvh = h / (a.heads / a.kv_heads), dim4 = (a.dim + 3) & ~3u, pieces = dim4 / 4;
    const uint32_t cl = warp * (32 / L) + lane / L, col0 = blockIdx.x * CC, col = col0 + cl;
    const bool col_ok = col < a.vdim;
    const float* pq = reinterpret_cast<const float*>(a.q) + (size_t)kvh * dim4;
    const float* pk = reinterpret_cast<const float*>(a.k) + (size_t)kvh * dim4;
    const float* pv = reinterpret_cast<const float*>(a.v) + (size_t)h * a.vdim + col0;
    const float* pg = reinterpret_cast<const float*>(a.decay) + h;
    const float* pb = reinterpret_cast<const float*>(a.beta) + h;
    const size_t qk_stride = (size_t)a.kv_heads * dim4, v_stride = (size_t)a.heads * a.vdim;
    auto stage = [&](uint32_t tb, uint32_t buf) {
        const uint32_t nb = tb < a.rows ? min((uint32_t)BATCH, a.rows - tb) : 0u;
        float* q = qs + buf * BATCH * ROWF;
        float* k = ks + buf * BATCH * ROWF;
        for (uint32_t i = tid; i < nb * pieces; i += GD_WARPS * 32) {
            const uint32_t r = i / pieces, c = (i - r * pieces) * 4;
            gd_cp_async16(q + r * ROWF + c, pq + (size_t)(tb + r) * qk_stride + c);
            gd_cp_async16(k + r * ROWF + c, pk + (size_t)(tb + r) * qk_stride + c);
        }
        for (uint32_t i = tid; i < nb * CC; i += GD_WARPS * 32) {
            const uint32_t r = i / CC, c = i % CC;
            if (col0 + c < a.vdim) gd_cp_async4(vs + (buf * BATCH + r) * CC + c, pv + (size_t)(tb + r) * v_stride + c);
        }
        if (tid < nb) {
            gd_cp_async4(gs + buf * BATCH + tid, pg + (size_t)(tb + tid) * a.heads);
            gd_cp_async4(bs + buf * BATCH + tid, pb + (size_t)(tb + tid) * a.heads);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (dim4 < (uint32_t)ROWF) {                     // channels past the head stay zero in both buffers
        const uint32_t tail = ROWF - dim4;
        for (uint32_t i = tid; i < 2 * BATCH * tail; i += GD_WARPS * 32) {
            const uint32_t r = i / tail, c = dim4 + i % tail;
            qs[r * ROWF + c] = 0.0f;
            ks[r * ROWF + c] = 0.0f;
        }
    }
    stage(0, 0);
    {   // the pass's last inputs of the convolution go to the ring (the launch before this one was its last reader)
        const uint32_t channels = 2 * a.kv_heads * a.dim + a.heads * a.vdim, prefix = gd_prefix(a), keep = min(a.rows, a.taps - 1);
        const uint32_t threads = gridDim.x * gridDim.y * blockDim.x, me = (blockIdx.y * gridDim.x + blockIdx.x) * blockDim.x + tid;
        const float* proj = reinterpret_cast<const float*>(a.proj);
        float* ring = reinterpret_cast<float*>(a.ring);
        for (uint32_t i = me; i < keep * channels; i += threads) {
            const uint32_t t = a.rows - keep + i / channels, c = i % channels;
            ring[(size_t)((prefix + t) % a.taps) * channels + c] = proj[(size_t)t * a.stride + c];
        }
    }
    float4 S[NV];
    float* state = reinterpret_cast<float*>(ga.state) + ((size_t)h * a.vdim + (col_ok ? col : 0u)) * dim4;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const uint32_t c = 4u * (i * L + part);
        S[i] = (col_ok && c < dim4) ? *reinterpret_cast<const float4*>(state + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    float* out = reinterpret_cast<float*>(ga.out) + (size_t)h * a.vdim + col;
    uint32_t buf = 0;
    for (uint32_t tb = 0; tb < a.rows; tb += BATCH, buf ^= 1) {
        const uint32_t nb = min((uint32_t)BATCH, a.rows - tb);
        stage(tb + BATCH, buf ^ 1);
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const float* q = qs + buf * BATCH * ROWF + part * 4;
        const float* k = ks + buf * BATCH * ROWF + part * 4;
        const float* v = vs + buf * BATCH * CC + cl;
        const float* g = gs + buf * BATCH;
        const float* b = bs + buf * BATCH;
        auto load_row = [&](float4 (&x)[NV], const float* row) {
#pragma unroll
            for (int i = 0; i < NV; ++i) x[i] = *reinterpret_cast<const float4*>(row + i * L * 4);
        };
        uint32_t r0 = 0;
        for (; r0 + U <= nb; r0 += U) {              // U tokens in straight-line code: the next token's rows are read during this token's reduction
            float gr[U], bg[U], bv[U], o[U];
            float4 kc[NV], qc[NV], kn[NV], qn[NV];
            load_row(kc, k + r0 * ROWF);
            load_row(qc, q + r0 * ROWF);
#pragma unroll
            for (int j = 0; j < U; ++j) {
                const float beta = b[r0 + j];
                gr[j] = g[r0 + j];
                bg[j] = -beta * gr[j];
                bv[j] = beta * v[(r0 + j) * CC];
            }
#pragma unroll
            for (int j = 0; j < U; ++j) {
                if (j + 1 < U) {
                    load_row(kn, k + (r0 + j + 1) * ROWF);
                    load_row(qn, q + (r0 + j + 1) * ROWF);
                }
                const float z = gd_lane_sum<L>(gd_dot<NV>(S, kc));
                gd_update<NV>(S, kc, gr[j], fmaf(bg[j], z, bv[j]));
                o[j] = gd_dot<NV>(S, qc);
                if (j + 1 < U) {
#pragma unroll
                    for (int i = 0; i < NV; ++i) { kc[i] = kn[i]; qc[i] = qn[i]; }
                }
            }
            // the U read-outs meet over the lanes of a column all at once: at every level a lane keeps half of the values
            gd_transpose_sum<U, L>(o, part);
            if (col_ok && part % (L / U) == 0) out[(size_t)(tb + r0 + part / (L / U)) * v_stride] = o[0];
        }
        for (; r0 < nb; ++r0) {
            float4 k4[NV], q4[NV];
            load_row(k4, k + r0 * ROWF);
            load_row(q4, q + r0 * ROWF);
            const float gr = g[r0], beta = b[r0];
            const float z = gd_lane_sum<L>(gd_dot<NV>(S, k4));
            gd_update<NV>(S, k4, gr, fmaf(-beta * gr, z, beta * v[r0 * CC]));
            const float o = gd_lane_sum<L>(gd_dot<NV>(S, q4));
            if (part == 0 && col_ok) out[(size_t)(tb + r0) * v_stride] = o;
        }
        __syncthreads();
    }
    if (col_ok) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4u * (i * L + part);
            if (c < dim4) *reinterpret_cast<float4*>(state + c) = S[i];
        }
    }
}

constexpr int GS_THREADS = 256;

// CL CTAs (one cluster) per head, ceil(vdim / CL) columns each, GS_THREADS / L columns at a time
template <int CL, int L, int NV>
__global__ void __cluster_dims__(CL, 1, 1) __launch_bounds__(GS_THREADS) gated_delta_step_kernel(const uzu_gated_delta_step_args sa) {
    constexpr int ROWF = L * NV * 4, CPP = GS_THREADS / L;
    extern __shared__ __align__(16) float gd_smem[];
    __shared__ float red_q[GS_THREADS / 32], red_k[GS_THREADS / 32], red_o[32], ss_parts[CL];
    const uzu_delta_prepare_args& a = sa.prep;
    pdl_launch_dependents();
    if constexpr (CL > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");     // "this CTA runs": awaited before the first remote store
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, part = tid % L;
    const uint32_t h = blockIdx.x / CL, rank = blockIdx.x % CL, group = a.heads / a.kv_heads, kvh = h / group;
    const uint32_t per = (a.vdim + CL - 1) / CL, col0 = min(a.vdim, rank * per), ncols = min(a.vdim, col0 + per) - col0;
    const uint32_t kd = a.kv_heads * a.dim, channels = 2 * kd + a.heads * a.vdim, dim4 = (a.dim + 3) & ~3u;
    float* qs = gd_smem;             // [ROWF]
    float* ks = qs + ROWF;           // [ROWF]
    float* vs = ks + ROWF;           // [per]
    float* os = vs + per;            // [per]
    float* state = reinterpret_cast<float*>(sa.state) + ((size_t)h * a.vdim + col0) * dim4;
    float4 S[NV];
    auto load_state = [&](uint32_t cl) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4u * (i * L + part);
            S[i] = (cl < ncols && c < dim4) ? *reinterpret_cast<const float4*>(state + (size_t)cl * dim4 + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
    };
    load_state(tid / L);             // nothing in front of this kernel writes the state or the ring: requested before the wait
    // ... and so is what the convolution takes from earlier tokens: all but the last tap
    const uint32_t prefix = gd_prefix(a), v0 = 2 * kd + h * a.vdim + col0;
    constexpr int QK = (2 * ROWF + GS_THREADS - 1) / GS_THREADS;      // q / k channels of a thread
    float qk_past[QK], qk_tap[QK], v_past = 0.0f, v_tap = 0.0f;
    auto qk_channel = [&](uint32_t i) { return (i < ROWF ? 0u : kd - ROWF) + kvh * a.dim + i; };      // (i counts q channels, then k channels)
    auto in_head = [&](uint32_t i) { return i < 2 * ROWF && (i < ROWF ? i : i - ROWF) < a.dim; };
#pragma unroll
    for (int u = 0; u < QK; ++u) {
        const uint32_t i = tid + u * GS_THREADS;
        qk_past[u] = qk_tap[u] = 0.0f;
        if (in_head(i)) gd_conv_past(a, channels, prefix, qk_channel(i), qk_past[u], qk_tap[u]);
    }
    if (tid < ncols) gd_conv_past(a, channels, prefix, v0 + tid, v_past, v_tap);
    const float a_log = reinterpret_cast<const float*>(a.a_log)[h], dt_bias = reinterpret_cast<const float*>(a.dt_bias)[h];
    const float norm0 = tid < ncols ? reinterpret_cast<const float*>(sa.norm)[(size_t)h * a.vdim + col0 + tid] : 0.0f;
    pdl_wait();
    const float* proj = reinterpret_cast<const float*>(a.proj);
    const float* gate = proj + sa.gate_offset + (size_t)h * a.vdim + col0;
    const float gate0 = tid < ncols ? gate[tid] : 0.0f;
    float* ring = reinterpret_cast<float*>(a.ring) + (size_t)(prefix % a.taps) * channels;        // the slot of this token: nobody reads it here
    float sq = 0.0f, sk = 0.0f;
#pragma unroll
    for (int u = 0; u < QK; ++u) {
        const uint32_t i = tid + u * GS_THREADS;
        float y = 0.0f;
        if (in_head(i)) {
            const float x = proj[qk_channel(i)];
            y = gd_silu(fmaf(qk_tap[u], x, qk_past[u]));
            if (rank == 0 && h % group == 0 && a.taps > 1) ring[qk_channel(i)] = x;
        }
        if (i < 2 * ROWF) qs[i] = y;                                     // ks follows qs
        if (i < ROWF) sq = fmaf(y, y, sq);
        else sk = fmaf(y, y, sk);
    }
    for (uint32_t i = tid; i < ncols; i += GS_THREADS) {
        if (i >= GS_THREADS) gd_conv_past(a, channels, prefix, v0 + i, v_past, v_tap);
        const float x = proj[v0 + i];
        vs[i] = gd_silu(fmaf(v_tap, x, v_past));
        if (a.taps > 1) ring[v0 + i] = x;
    }
    const float g = gd_decay(a_log, proj[a.a_offset + h] + dt_bias);
    const float beta = gd_sigmoid(proj[a.b_offset + h]);
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) { red_q[warp] = sq; red_k[warp] = sk; }
    __syncthreads();
    float tq = 0.0f, tk = 0.0f;
#pragma unroll
    for (int w = 0; w < GS_THREADS / 32; ++w) { tq += red_q[w]; tk += red_k[w]; }
    const float fq = (1.0f / sqrtf(tq + kUnitEps)) * (1.0f / sqrtf((float)a.dim)), fk = 1.0f / sqrtf(tk + kUnitEps);
    float4 q4[NV], k4[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const float4 q = *reinterpret_cast<const float4*>(qs + 4 * (i * L + part)), k = *reinterpret_cast<const float4*>(ks + 4 * (i * L + part));
        q4[i] = make_float4(q.x * fq, q.y * fq, q.z * fq, q.w * fq);
        k4[i] = make_float4(k.x * fk, k.y * fk, k.z * fk, k.w * fk);
    }
    for (uint32_t cb = 0; cb < ncols; cb += CPP) {
        const uint32_t cl = cb + tid / L;
        if (cb) load_state(cl);
        const float z = gd_lane_sum<L>(gd_dot<NV>(S, k4));
        const float u = beta * ((cl < ncols ? vs[cl] : 0.0f) - g * z);
        gd_update<NV>(S, k4, g, u);
        const float o = gd_lane_sum<L>(gd_dot<NV>(S, q4));
        if (cl < ncols) {
            if (part == 0) os[cl] = o;
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const uint32_t c = 4u * (i * L + part);
                if (c < dim4) *reinterpret_cast<float4*>(state + (size_t)cl * dim4 + c) = S[i];
            }
        }
    }
    __syncthreads();
    float ss = 0.0f;
    for (uint32_t i = tid; i < ncols; i += GS_THREADS) ss = fmaf(os[i], os[i], ss);
    ss = block_sum(ss, red_o);
    if constexpr (CL > 1) {
        asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
        if (tid < CL) {
            const uint32_t local = (uint32_t)__cvta_generic_to_shared(&ss_parts[rank]);
            uint32_t remote;
            asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"(tid));
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(remote), "f"(ss) : "memory");
        }
        asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
        ss = 0.0f;
#pragma unroll
        for (int c = 0; c < CL; ++c) ss += ss_parts[c];
    }
    const float inv = 1.0f / sqrtf(ss / (float)a.vdim + sa.epsilon);
    float* out = reinterpret_cast<float*>(sa.out) + (size_t)h * a.vdim + col0;
    if (tid < ncols) out[tid] = os[tid] * inv * norm0 * gd_silu(gate0);
    const float* norm = reinterpret_cast<const float*>(sa.norm) + (size_t)h * a.vdim + col0;
    for (uint32_t i = tid + GS_THREADS; i < ncols; i += GS_THREADS) out[i] = os[i] * inv * norm[i] * gd_silu(gate[i]);
}

static const char* delta_prepare_check(const uzu_delta_prepare_args& a, bool scratch) {
    if (!a.proj || !a.conv || !a.ring || !a.a_log || !a.dt_bias || (scratch && (!a.q || !a.k || !a.v || !a.decay || !a.beta))) return "null operand";
    if (a.heads == 0 || a.kv_heads == 0 || a.heads % a.kv_heads || a.dim == 0 || a.dim > 1024 || a.vdim == 0 || a.vdim > 4096 || a.taps == 0)
        return "kv_heads must divide heads, dim must be in 1..1024, vdim in 1..4096, taps positive";
    if (scratch && ((a.q & 15) || (a.k & 15))) return "the q / k rows must be 16-byte aligned";
    const uint64_t channels = 2ull * a.kv_heads * a.dim + (uint64_t)a.heads * a.vdim;
    if (a.stride < channels || a.a_offset + a.heads > a.stride || a.b_offset + a.heads > a.stride) return "a projection row is shorter than its parts";
    return nullptr;
}

// lanes per value column and float4 of key channels per lane, by head size
template <typename F>
static void by_key_size(uint32_t dim, F&& f) {
    if (dim <= 32) f(std::integral_constant<int, 8>{}, std::integral_constant<int, 1>{});
    else if (dim <= 64) f(std::integral_constant<int, 8>{}, std::integral_constant<int, 2>{});
    else if (dim <= 128) f(std::integral_constant<int, 8>{}, std::integral_constant<int, 4>{});
    else if (dim <= 256) f(std::integral_constant<int, 16>{}, std::integral_constant<int, 4>{});
    else if (dim <= 512) f(std::integral_constant<int, 32>{}, std::integral_constant<int, 4>{});
    else f(std::integral_constant<int, 32>{}, std::integral_constant<int, 8>{});
}

}  // namespace uzu

extern "C" {
using namespace uzu;

void uzu_delta_prepare_encode(uzu_command_buffer* cmd, const uzu_delta_prepare_args* a) {
    if (!encodable(cmd, "delta_prepare")) return;
    if (const char* err = delta_prepare_check(*a, true)) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, std::string("delta_prepare: ") + err);
        return;
    }
    if (a->rows == 0) return;
    const uint32_t units = 2 * a->kv_heads + a->heads + 1, widest = std::max(a->dim, a->vdim);
    if (a->rows >= 4 && a->taps >= 2 && a->taps <= 4 && widest <= 256) {
        const uint32_t blocks = (a->rows + GP_ROWS - 1) / GP_ROWS;
        auto go = [&](auto kernel) { launch(cmd, "delta_prepare_kernel", kernel, dim3((blocks * units + 3) / 4), dim3(128), 0, *a); };
        auto by_width = [&](auto taps_c) {
            constexpr int T = decltype(taps_c)::value;
            if (widest <= 32) go(delta_prepare_window_kernel<T, 1>);
            else if (widest <= 64) go(delta_prepare_window_kernel<T, 2>);
            else if (widest <= 128) go(delta_prepare_window_kernel<T, 4>);
            else go(delta_prepare_window_kernel<T, 8>);
        };
        if (a->taps == 2) by_width(std::integral_constant<int, 2>{});
        else if (a->taps == 3) by_width(std::integral_constant<int, 3>{});
        else by_width(std::integral_constant<int, 4>{});
        return;
    }
    const uint32_t items = a->rows * units;
    launch(cmd, "delta_prepare_kernel", delta_prepare_kernel, dim3((items + 3) / 4), dim3(128), 0, *a);
}

void uzu_gated_delta_encode(uzu_command_buffer* cmd, const uzu_gated_delta_args* a) {
    if (!encodable(cmd, "gated_delta")) return;
    const char* err = delta_prepare_check(a->prep, true);
    if (!err && (!a->state || !a->out || (a->state & 15))) err = "null or unaligned state, or null output";
    if (err) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, std::string("gated_delta: ") + err);
        return;
    }
    if (a->prep.rows == 0) return;
    by_key_size(a->prep.dim, [&](auto l_c, auto nv_c) {
        constexpr int L = decltype(l_c)::value, NV = decltype(nv_c)::value, CC = GD_WARPS * (32 / L), BATCH = gd_batch<L, NV>();
        constexpr size_t smem = ((size_t)4 * BATCH * L * NV * 4 + (size_t)2 * BATCH * CC + 4 * BATCH) * sizeof(float);
        static std::atomic<uint64_t> done{0};
        if (smem > 48 * 1024) opt_in_dynamic_smem(cmd, gated_delta_kernel<L, NV>, (int)smem, done);
        launch(cmd, "gated_delta_kernel", gated_delta_kernel<L, NV>, dim3((a->prep.vdim + CC - 1) / CC, a->prep.heads), dim3(GD_WARPS * 32), smem, *a);
    });
}

void uzu_gated_delta_step_encode(uzu_command_buffer* cmd, const uzu_gated_delta_step_args* a) {
    if (!encodable(cmd, "gated_delta_step")) return;
    const char* err = delta_prepare_check(a->prep, false);
    if (!err && (!a->state || !a->out || !a->norm || (a->state & 15))) err = "null operand or unaligned state";
    if (!err && a->prep.rows != 1) err = "one token per launch";
    if (!err && (uint64_t)a->gate_offset + (uint64_t)a->prep.heads * a->prep.vdim > a->prep.stride) err = "a projection row is shorter than its parts";
    if (err) {
        cmd->record_error(UZU_ERROR_INVALID_ARGUMENT, std::string("gated_delta_step: ") + err);
        return;
    }
    by_key_size(a->prep.dim, [&](auto l_c, auto nv_c) {
        constexpr int L = decltype(l_c)::value, NV = decltype(nv_c)::value;
        auto go = [&](auto cl_c) {
            constexpr int CL = decltype(cl_c)::value;
            const size_t smem = ((size_t)2 * L * NV * 4 + (size_t)2 * ((a->prep.vdim + CL - 1) / CL)) * sizeof(float);
            launch(cmd, "gated_delta_step_kernel", gated_delta_step_kernel<CL, L, NV>, dim3(a->prep.heads * CL), dim3(GS_THREADS), smem, *a);
        };
        // one pass over a CTA's columns where a cluster of four can do that; a head of few columns needs no cluster
        if (a->prep.vdim > (uint32_t)(GS_THREADS / L)) go(std::integral_constant<int, 4>{});
        else go(std::integral_constant<int, 1>{});
    });
}

}  // extern "C"
