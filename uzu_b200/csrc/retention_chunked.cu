// Retention over long passes in chunks of 64 tokens, on the tensor pipe. Per head with decay g, chunk rows i, j = 0 .. n-1 and the state S before it:
//   o_i = g^(i+1) S^T q_i + sum_(j <= i) g^(i-j) (q_i . k_j) v_j,       S' = g^n S + sum_j g^(n-1-j) k_j v_j^T
// Three launches: (1) every chunk's own sum of k v^T, all chunks at once; (2) a scan over the chunks, element by element of the state, which leaves
// the state before every chunk; (3) the outputs, all chunks at once. mma.sync.m16n8k16 (bf16 x bf16 -> f32):
//   q, k and v are rounded to bf16 once (after their silu); everything that carries a decay or is a sum of others -- the decayed keys of (1), the
//   states, the decayed scores -- is taken as hi + lo, two bf16 numbers per f32 entry, so its rounding stays below 2^-16. States, sums and decays are f32.
// The scratch holds f32 sums after (1) and the states before the chunks as packed (hi, lo) pairs after (2).
#include "common.cuh"

namespace uzu {

namespace {

constexpr int RC_ROWS = 64, RC_COLS = 64, RC_PAD = 8;        // tokens of a chunk, value columns of a CTA
constexpr int RC_THREADS = 256;

__device__ __forceinline__ void rc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <bool TRANS>
__device__ __forceinline__ void rc_ldmatrix(uint32_t (&r)[4], const void* smem_ptr) {
    const uint32_t addr = (uint32_t)__cvta_generic_to_shared(smem_ptr);
    if constexpr (TRANS)
        asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
    else
        asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

__device__ __forceinline__ uint32_t rc_pack(float x0, float x1) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x0, x1);
    return *reinterpret_cast<const uint32_t*>(&h);
}

// x = hi + lo with both parts bf16; two values packed for a fragment or a shared-memory word
__device__ __forceinline__ void rc_split(float x0, float x1, uint32_t& hi, uint32_t& lo) {
    hi = rc_pack(x0, x1);
    lo = rc_pack(x0 - __uint_as_float(hi << 16), x1 - __uint_as_float(hi & 0xffff0000u));
}

// (the fast exponential and division are good to about 2^-20; the result is rounded to bf16 next)
__device__ __forceinline__ float rc_input(uint32_t op, float x) { return op == 1 ? __fdividef(x, 1.0f + __expf(-x)) : x; }

__device__ __forceinline__ float4 rc_input4(uint32_t op, float4 x) {
    return make_float4(rc_input(op, x.x), rc_input(op, x.y), rc_input(op, x.z), rc_input(op, x.w));
}

// rows [0, n) of `cols` f32 columns (a multiple of 4) -> bf16 rows of `ld`; rows from n to RC_ROWS are zero
template <int BATCH, typename F>
__device__ __forceinline__ void rc_stage(const float* src, size_t stride, uint32_t cols, uint32_t n, F&& store) {
    const uint32_t c4 = cols / 4, total = RC_ROWS * c4;
    for (uint32_t i0 = threadIdx.x; i0 < total; i0 += BATCH * blockDim.x) {
        float4 x[BATCH];
#pragma unroll
        for (int u = 0; u < BATCH; ++u) {
            const uint32_t i = i0 + u * blockDim.x, r = i / c4, c = (i - r * c4) * 4;
            x[u] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (i < total && r < n) x[u] = *reinterpret_cast<const float4*>(src + (size_t)r * stride + c);
        }
#pragma unroll
        for (int u = 0; u < BATCH; ++u) {
            const uint32_t i = i0 + u * blockDim.x, r = i / c4, c = (i - r * c4) * 4;
            if (i < total) store(r, c, x[u]);
        }
    }
}

}  // namespace

// (1) scratch[head, chunk] = sum_j g^(n-1-j) k_j v_j^T.  M = key channels (16 per warp), N = 64 value columns, K = tokens.
__global__ void __launch_bounds__(RC_THREADS) retention_chunk_sums_kernel(const uzu_retention_args a) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char rc_raw[];
    __shared__ float power[RC_ROWS];
    const uint32_t dim = a.dim, vdim = a.vdim, ldk = dim + RC_PAD, ldv = RC_COLS + RC_PAD;
    __nv_bfloat16* k_hi = reinterpret_cast<__nv_bfloat16*>(rc_raw);          // [64][ldk]
    __nv_bfloat16* k_lo = k_hi + RC_ROWS * ldk;
    __nv_bfloat16* v_s = k_lo + RC_ROWS * ldk;                               // [64][ldv]
    const uint32_t chunk = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * RC_COLS, chunks = gridDim.x;
    const uint32_t t0 = chunk * RC_ROWS, n = min((uint32_t)RC_ROWS, a.rows - t0), cols = min((uint32_t)RC_COLS, vdim - v0);
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
    if (tid < RC_ROWS) power[tid] = tid < n ? powf(reinterpret_cast<const float*>(a.decay)[head], (float)(n - 1 - tid)) * a.key_scale : 0.0f;
    pdl_wait();
    __syncthreads();
    const float* k = reinterpret_cast<const float*>(a.k) + (size_t)t0 * a.k_stride + (size_t)head * dim;
    const float* v = reinterpret_cast<const float*>(a.v) + (size_t)t0 * a.v_stride + (size_t)head * vdim + v0;
    rc_stage<8>(k, a.k_stride, dim, n, [&](uint32_t r, uint32_t c, float4 x) {
        x = rc_input4(a.input_op, x);
        const float p = power[r];
        uint2 hi, lo;
        // (the rounding of k itself comes first: the outputs meet the same rounded keys)
        const uint32_t r0 = rc_pack(x.x, x.y), r1 = rc_pack(x.z, x.w);
        rc_split(__uint_as_float(r0 << 16) * p, __uint_as_float(r0 & 0xffff0000u) * p, hi.x, lo.x);
        rc_split(__uint_as_float(r1 << 16) * p, __uint_as_float(r1 & 0xffff0000u) * p, hi.y, lo.y);
        *reinterpret_cast<uint2*>(k_hi + r * ldk + c) = hi;
        *reinterpret_cast<uint2*>(k_lo + r * ldk + c) = lo;
    });
    rc_stage<8>(v, a.v_stride, cols, n, [&](uint32_t r, uint32_t c, float4 x) {
        x = rc_input4(a.input_op, x);
        *reinterpret_cast<uint2*>(v_s + r * ldv + c) = make_uint2(rc_pack(x.x, x.y), rc_pack(x.z, x.w));
    });
    __syncthreads();
    if (warp * 16 >= dim) return;
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[j][c] = 0.0f;
    const uint32_t nblocks = cols / 16;
#pragma unroll
    for (int kk = 0; kk < RC_ROWS / 16; ++kk) {
        uint32_t b[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if ((uint32_t)j < nblocks) rc_ldmatrix<true>(b[j], v_s + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + (lane >> 4) * 8 + j * 16);
        uint32_t hi[4], lo[4];
        const uint32_t at = (kk * 16 + (lane & 7) + (lane >> 4) * 8) * ldk + warp * 16 + ((lane >> 3) & 1) * 8;
        rc_ldmatrix<true>(hi, k_hi + at);
        rc_ldmatrix<true>(lo, k_lo + at);
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if ((uint32_t)j < 2 * nblocks) rc_mma(acc[j], hi, b[j >> 1][(j & 1) * 2], b[j >> 1][(j & 1) * 2 + 1]);
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if ((uint32_t)j < 2 * nblocks) rc_mma(acc[j], lo, b[j >> 1][(j & 1) * 2], b[j >> 1][(j & 1) * 2 + 1]);
    }
    float* out = reinterpret_cast<float*>(a.chunk_scratch) + ((size_t)head * chunks + chunk) * dim * vdim + v0;
#pragma unroll
    for (int j = 0; j < 8; ++j)
        if ((uint32_t)j < 2 * nblocks) {
            float* o = out + (size_t)(warp * 16 + g) * vdim + j * 8 + t4 * 2;
            *reinterpret_cast<float2*>(o) = make_float2(acc[j][0], acc[j][1]);
            *reinterpret_cast<float2*>(o + (size_t)8 * vdim) = make_float2(acc[j][2], acc[j][3]);
        }
}

// (2) four state elements per thread: the sums become the states before their chunks (hi in the upper half of a word), the last state is stored
__global__ void __launch_bounds__(256) retention_chunk_scan_kernel(const uzu_retention_args a) {
    pdl_launch_dependents();
    const uint32_t head = blockIdx.y, chunks = (a.rows + RC_ROWS - 1) / RC_ROWS, last = a.rows - (chunks - 1) * RC_ROWS;
    const size_t size4 = (size_t)a.dim * a.vdim / 4, i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const float decay = reinterpret_cast<const float*>(a.decay)[head];
    const float whole = powf(decay, (float)RC_ROWS), part = powf(decay, (float)last);
    pdl_wait();
    if (i >= size4) return;
    float4* state = reinterpret_cast<float4*>(a.state) + head * size4 + i;
    float4* u = reinterpret_cast<float4*>(a.chunk_scratch) + (size_t)head * chunks * size4 + i;
    float4 s = *state;
    constexpr int AHEAD = 8;
    float4 x[AHEAD];
#pragma unroll
    for (int q = 0; q < AHEAD; ++q)
        if ((uint32_t)q < chunks) x[q] = u[q * size4];
    auto word = [](float v) {
        const __nv_bfloat16 h = __float2bfloat16_rn(v), l = __float2bfloat16_rn(v - __bfloat162float(h));
        return ((uint32_t)__bfloat16_as_ushort(h) << 16) | __bfloat16_as_ushort(l);
    };
    for (uint32_t c0 = 0; c0 < chunks; c0 += AHEAD) {
#pragma unroll
        for (int q = 0; q < AHEAD; ++q) {
            const uint32_t c = c0 + q;
            if (c < chunks) {
                const float d = c + 1 == chunks ? part : whole;
                const float4 add = x[q];
                if (c + AHEAD < chunks) x[q] = u[(c + AHEAD) * size4];
                *reinterpret_cast<uint4*>(u + c * size4) = make_uint4(word(s.x), word(s.y), word(s.z), word(s.w));
                s = make_float4(fmaf(d, s.x, add.x), fmaf(d, s.y, add.y), fmaf(d, s.z, add.z), fmaf(d, s.w, add.w));
            }
        }
    }
    *state = s;
}

// (3) 64 tokens x 64 value columns of one head; a warp takes 16 tokens and half of the columns
__global__ void __launch_bounds__(RC_THREADS, 2) retention_chunk_out_kernel(const uzu_retention_args a) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char rc_raw[];
    __shared__ float power[RC_ROWS + 1];
    const uint32_t dim = a.dim, vdim = a.vdim, ldk = dim + RC_PAD, ldv = RC_COLS + RC_PAD;
    __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(rc_raw);           // [64][ldk]
    __nv_bfloat16* k_s = q_s + RC_ROWS * ldk;                                // [64][ldk]
    __nv_bfloat16* v_s = k_s + RC_ROWS * ldk;                                // [64][ldv]
    __nv_bfloat16* s_hi = v_s + RC_ROWS * ldv;                               // [dim][ldv]
    __nv_bfloat16* s_lo = s_hi + dim * ldv;
    const uint32_t chunk = blockIdx.x, head = blockIdx.y, v0 = blockIdx.z * RC_COLS, chunks = gridDim.x;
    const uint32_t t0 = chunk * RC_ROWS, n = min((uint32_t)RC_ROWS, a.rows - t0), cols = min((uint32_t)RC_COLS, vdim - v0);
    const uint32_t tid = threadIdx.x, lane = tid & 31, warp = (tid >> 5) & 3, part = tid >> 7, g = lane >> 2, t4 = lane & 3;
    if (tid <= RC_ROWS) power[tid] = powf(reinterpret_cast<const float*>(a.decay)[head], (float)tid);
    pdl_wait();
    auto to_bf16 = [&](__nv_bfloat16* tile, uint32_t ld) {
        return [tile, ld, op = a.input_op](uint32_t r, uint32_t c, float4 x) {
            x = rc_input4(op, x);
            *reinterpret_cast<uint2*>(tile + r * ld + c) = make_uint2(rc_pack(x.x, x.y), rc_pack(x.z, x.w));
        };
    };
    rc_stage<8>(reinterpret_cast<const float*>(a.q) + (size_t)t0 * a.q_stride + (size_t)head * dim, a.q_stride, dim, n, to_bf16(q_s, ldk));
    rc_stage<8>(reinterpret_cast<const float*>(a.k) + (size_t)t0 * a.k_stride + (size_t)head * dim, a.k_stride, dim, n, to_bf16(k_s, ldk));
    rc_stage<8>(reinterpret_cast<const float*>(a.v) + (size_t)t0 * a.v_stride + (size_t)head * vdim + v0, a.v_stride, cols, n, to_bf16(v_s, ldv));
    {
        const uint32_t* src = reinterpret_cast<const uint32_t*>(a.chunk_scratch) + ((size_t)head * chunks + chunk) * dim * vdim + v0;
        const uint32_t c4 = cols / 4, total = dim * c4;
        constexpr int BATCH = 8;
        for (uint32_t i0 = tid; i0 < total; i0 += BATCH * RC_THREADS) {
            uint4 x[BATCH];
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                const uint32_t i = i0 + u * RC_THREADS, r = i / c4, c = (i - r * c4) * 4;
                if (i < total) x[u] = *reinterpret_cast<const uint4*>(src + (size_t)r * vdim + c);
            }
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                const uint32_t i = i0 + u * RC_THREADS, r = i / c4, c = (i - r * c4) * 4;
                if (i < total) {
                    const uint4 w = x[u];
                    *reinterpret_cast<uint2*>(s_hi + r * ldv + c) = make_uint2((w.x >> 16) | (w.y & 0xffff0000u), (w.z >> 16) | (w.w & 0xffff0000u));
                    *reinterpret_cast<uint2*>(s_lo + r * ldv + c) = make_uint2((w.x & 0xffffu) | (w.y << 16), (w.z & 0xffffu) | (w.w << 16));
                }
            }
        }
    }
    __syncthreads();
    const uint32_t c_first = part * (RC_COLS / 2);              // this warp's columns
    if (c_first >= cols) return;
    float o[4][4], s[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) { s[j][c] = 0.0f; if (j < 4) o[j][c] = 0.0f; }
    const uint32_t dk = dim / 16, nblocks = min((uint32_t)RC_COLS / 2, cols - c_first) / 16, row_lo = warp * 16 + g;
    // what the state before the chunk gives, and the scores of the chunk's own keys (only those up to the warp's last token)
    for (uint32_t kk = 0; kk < dk; ++kk) {
        uint32_t q[4];
        rc_ldmatrix<false>(q, q_s + (warp * 16 + (lane & 15)) * ldk + kk * 16 + (lane >> 4) * 8);
        const uint32_t at = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + (lane >> 4) * 8 + c_first;
        uint32_t b[2][4], bl[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
            if ((uint32_t)j < nblocks) {
                rc_ldmatrix<true>(b[j], s_hi + at + j * 16);
                rc_ldmatrix<true>(bl[j], s_lo + at + j * 16);
            }
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if ((uint32_t)j < 2 * nblocks) rc_mma(o[j], q, b[j >> 1][(j & 1) * 2], b[j >> 1][(j & 1) * 2 + 1]);
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if ((uint32_t)j < 2 * nblocks) rc_mma(o[j], q, bl[j >> 1][(j & 1) * 2], bl[j >> 1][(j & 1) * 2 + 1]);
        // keys: two tiles of 8 tokens per load: (tokens 0-7, channels 0-7), (0-7, 8-15), (8-15, 0-7), (8-15, 8-15)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            if ((uint32_t)j <= warp) {
                uint32_t kb[4];
                rc_ldmatrix<false>(kb, k_s + (j * 16 + (lane & 7) + ((lane >> 4) << 3)) * ldk + kk * 16 + ((lane >> 3) & 1) * 8);
                rc_mma(s[2 * j], q, kb[0], kb[1]);
                rc_mma(s[2 * j + 1], q, kb[2], kb[3]);
            }
        }
    }
    const float key_scale = a.key_scale;
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const uint32_t i = row_lo + 8 * (c >> 1), t = j * 8 + t4 * 2 + (c & 1);
            if (j < 4) o[j][c] *= power[i + 1];
            s[j][c] = t <= i ? s[j][c] * (power[i - t] * key_scale) : 0.0f;
        }
#pragma unroll
    for (int kk = 0; kk < RC_ROWS / 16; ++kk) {
        if ((uint32_t)kk > warp) continue;                 // all of these tokens come after the warp's
        uint32_t ph[4], pl[4];
        rc_split(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]);
        rc_split(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
        rc_split(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]);
        rc_split(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
        uint32_t b[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
            if ((uint32_t)j < nblocks) rc_ldmatrix<true>(b[j], v_s + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + (lane >> 4) * 8 + c_first + j * 16);
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if ((uint32_t)j < 2 * nblocks) rc_mma(o[j], ph, b[j >> 1][(j & 1) * 2], b[j >> 1][(j & 1) * 2 + 1]);
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if ((uint32_t)j < 2 * nblocks) rc_mma(o[j], pl, b[j >> 1][(j & 1) * 2], b[j >> 1][(j & 1) * 2 + 1]);
    }
    const float qscale = a.query_scale != 0.0f ? a.query_scale : 1.0f;
    float* out = reinterpret_cast<float*>(a.out) + (size_t)t0 * a.out_stride + (size_t)head * vdim + v0 + c_first;
#pragma unroll
    for (int j = 0; j < 4; ++j)
        if ((uint32_t)j < 2 * nblocks) {
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const uint32_t r = row_lo + 8 * half;
                if (r < n) *reinterpret_cast<float2*>(out + (size_t)r * a.out_stride + j * 8 + t4 * 2) = make_float2(o[j][2 * half] * qscale, o[j][2 * half + 1] * qscale);
            }
        }
}

// Passes of >= 64 tokens with a scratch, one decay per head, head sizes that are multiples of 16 up to 128 (keys) and 256 (values), 16-byte aligned
// rows. Everything else runs token by token.
bool encode_retention_chunked(uzu_command_buffer* cmd, const uzu_retention_args& a) {
    static const bool off = getenv("UZU_RETENTION_NO_CHUNKS") != nullptr;       // A/B runs
    if (off || !a.chunk_scratch || a.token_decay || a.rows < (uint32_t)RC_ROWS || a.dim % 16 || a.vdim % 16 || a.dim > 128 || a.vdim > 256) return false;
    if ((a.q | a.k | a.v | a.chunk_scratch | a.state) & 15 || (a.out & 7) || a.q_stride % 4 || a.k_stride % 4 || a.v_stride % 4 || a.out_stride % 2) return false;
    const uint32_t chunks = (a.rows + RC_ROWS - 1) / RC_ROWS, tiles = (a.vdim + RC_COLS - 1) / RC_COLS;
    const size_t row_k = (a.dim + RC_PAD) * sizeof(__nv_bfloat16), row_v = (RC_COLS + RC_PAD) * sizeof(__nv_bfloat16), most_k = (128 + RC_PAD) * sizeof(__nv_bfloat16);
    static std::atomic<uint64_t> done[2];
    opt_in_dynamic_smem(cmd, retention_chunk_sums_kernel, (int)(RC_ROWS * (2 * most_k + row_v)), done[0]);
    opt_in_dynamic_smem(cmd, retention_chunk_out_kernel, (int)(RC_ROWS * (2 * most_k + row_v) + 2 * 128 * row_v), done[1]);
    const dim3 grid(chunks, a.heads, tiles);
    launch(cmd, "retention_chunk_sums_kernel", retention_chunk_sums_kernel, grid, dim3(RC_THREADS), RC_ROWS * (2 * row_k + row_v), a);
    launch(cmd, "retention_chunk_scan_kernel", retention_chunk_scan_kernel, dim3((unsigned)(((size_t)a.dim * a.vdim / 4 + 255) / 256), a.heads), dim3(256), 0, a);
    launch(cmd, "retention_chunk_out_kernel", retention_chunk_out_kernel, grid, dim3(RC_THREADS), RC_ROWS * (2 * row_k + row_v) + 2 * a.dim * row_v, a);
    return true;
}

}  // namespace uzu
