// Memory-bound kernels of the step: embedding gather, residual-add + RMSNorm, rotation table,
// per-head QK RMSNorm + rotary + key/value write into pages, gated activation.
//
// All arithmetic is 32-bit and each result is rounded once into the activation dtype.  The
// residual stream itself is kept in 32-bit in both precisions.
#include "common.cuh"

using namespace mrun;

// ------------------------------------------------------------------------------------------
// Embedding: out[t, :] = float(table[ids[t], :]).  An id outside [0, vocab) gives a zero row;
// the host checks ids before the step, this only keeps the kernel inside the table.
// Reference call site: crates/mrun-engine/src/load.rs:330-335.
// ------------------------------------------------------------------------------------------
template <typename TW>
__global__ void embed_kernel(const TW* __restrict__ table, const int* __restrict__ ids,
                             float* __restrict__ out, int hidden, int vocab) {
    const int t = blockIdx.x;
    const int id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    const TW* row = table + (size_t)(ok ? id : 0) * hidden;
    float* dst = out + (size_t)t * hidden;
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) dst[h] = ok ? to_float(row[h]) : 0.f;
}

// Eight features a thread (a width that is a multiple of 8): a row is many threads' work, so that a step of a
// few tokens is not one thread's chain of loads.
template <typename TW>
__global__ void __launch_bounds__(128)
embed_vec_kernel(const TW* __restrict__ table, const int* __restrict__ ids, float* __restrict__ out, int hidden, int vocab) {
    const int t = blockIdx.x, c = (blockIdx.y * 128 + threadIdx.x) * 8;
    if (c >= hidden) return;
    const int id = ids[t];
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (id >= 0 && id < vocab) Vec8<TW>::load(table + (size_t)id * hidden + c, v);
    Vec8<float>::store(out + (size_t)t * hidden + c, v);
}

MRUN_API int mrun_embed(const void* table, int table_dtype, const int* ids, float* out, int tokens,
                        int hidden, int vocab, cudaStream_t stream) {
    MRUN_REQUIRE(tokens >= 0 && hidden > 0 && vocab > 0, "embed: bad sizes tokens=%d hidden=%d vocab=%d",
                 tokens, hidden, vocab);
    if (tokens == 0) return 0;
    if (hidden % 8 == 0 && (((uintptr_t)table | (uintptr_t)out) & 15) == 0 && (table_dtype == MRUN_F32 || table_dtype == MRUN_BF16)) {
        const dim3 grid(tokens, (hidden / 8 + 127) / 128);
        if (table_dtype == MRUN_F32)
            embed_vec_kernel<float><<<grid, 128, 0, stream>>>((const float*)table, ids, out, hidden, vocab);
        else
            embed_vec_kernel<__nv_bfloat16><<<grid, 128, 0, stream>>>((const __nv_bfloat16*)table, ids, out, hidden, vocab);
        MRUN_CHECK_LAUNCH("embed");
        return 0;
    }
    if (table_dtype == MRUN_F32)
        embed_kernel<float><<<tokens, 256, 0, stream>>>((const float*)table, ids, out, hidden, vocab);
    else if (table_dtype == MRUN_BF16)
        embed_kernel<__nv_bfloat16><<<tokens, 256, 0, stream>>>((const __nv_bfloat16*)table, ids, out,
                                                                 hidden, vocab);
    else
        return mrun_set_error("embed: unknown dtype code %d", table_dtype);
    MRUN_CHECK_LAUNCH("embed");
    return 0;
}

// ------------------------------------------------------------------------------------------
// Residual add + RMSNorm.
//   v = resid[src] + delta[src]   (delta may be null; 32-bit or of out's type)
//                  + share[src] * extra[src]   (a second branch with one factor a row, or null)
//   if rows == null: resid[src] = v            (the stream advances)
//   out[r] = v * rsqrt(mean(v^2) + eps) * weight
// With `rows` the kernel reads row rows[r] and leaves the stream untouched (final norm at the
// wanted positions only).  eps is added to the mean of squares
// (crates/mrun-engine/src/models/gated_delta.rs:11-13 states the form).
// One block of 256 threads per row whatever the batch, so the order of additions is fixed.
// ------------------------------------------------------------------------------------------
template <typename TA, typename TD>
__global__ void add_rmsnorm_kernel(float* __restrict__ resid, const TD* __restrict__ delta,
                                   const float* __restrict__ weight, float eps, TA* __restrict__ out,
                                   const int* __restrict__ rows, int hidden, const TA* __restrict__ extra,
                                   const float* __restrict__ share) {
    extern __shared__ float row_buf[];
    __shared__ float scratch[33];
    const int r = blockIdx.x;
    const int row = rows ? rows[r] : r;
    const size_t src = (size_t)row * hidden;
    const float part = extra ? share[row] : 0.f;
    const bool moved = delta || part != 0.f;
    float ss = 0.f;
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
        float v = resid[src + h];
        if (delta) v += to_float(delta[src + h]);
        if (part != 0.f) v = fmaf(part, to_float(extra[src + h]), v);
        row_buf[h] = v;
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float inv = rsqrtf(ss / (float)hidden + eps);
    TA* dst = out + (size_t)r * hidden;
    for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
        const float v = row_buf[h];
        if (!rows && moved) resid[src + h] = v;
        dst[h] = from_float<TA>(v * inv * weight[h]);
    }
}

// The same operation for widths that are a multiple of 8 and at most 8192: every thread keeps up
// to four 8-element chunks in registers and moves them with 16-byte loads and stores, so a row
// takes one pass and the latency of a few independent loads.  One block of 256 threads per row
// whatever the batch: the order of additions depends on the width only.
template <typename TA, typename TD>
__global__ void __launch_bounds__(256)
add_rmsnorm_vec_kernel(float* __restrict__ resid, const TD* __restrict__ delta,
                       const float* __restrict__ weight, float eps, TA* __restrict__ out,
                       const int* __restrict__ rows, int hidden, const TA* __restrict__ extra,
                       const float* __restrict__ share) {
    __shared__ float scratch[33];
    const int r = blockIdx.x;
    const int row = rows ? rows[r] : r;
    const size_t src = (size_t)row * hidden;
    const float part = extra ? share[row] : 0.f;
    const bool moved = delta || part != 0.f;
    const int chunks = hidden >> 3;
    float v[4][8];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int c = threadIdx.x + i * 256;
        if (c < chunks) {
            Vec8<float>::load(resid + src + c * 8, v[i]);
            if (delta) {
                float d[8];
                Vec8<TD>::load(delta + src + c * 8, d);
#pragma unroll
                for (int e = 0; e < 8; ++e) v[i][e] += d[e];
            }
            if (part != 0.f) {
                float d[8];
                Vec8<TA>::load(extra + src + c * 8, d);
#pragma unroll
                for (int e = 0; e < 8; ++e) v[i][e] = fmaf(part, d[e], v[i][e]);
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) ss += v[i][e] * v[i][e];
        }
    }
    ss = block_sum(ss, scratch);
    const float inv = rsqrtf(ss / (float)hidden + eps);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int c = threadIdx.x + i * 256;
        if (c < chunks) {
            if (!rows && moved) Vec8<float>::store(resid + src + c * 8, v[i]);
            float w[8], y[8];
            Vec8<float>::load(weight + c * 8, w);
#pragma unroll
            for (int e = 0; e < 8; ++e) y[e] = v[i][e] * inv * w[e];
            Vec8<TA>::store(out + (size_t)r * hidden + c * 8, y);
        }
    }
}

template <typename TA, typename TD>
static int launch_add_rmsnorm(float* resid, const void* delta, const float* weight, float eps, void* out,
                              const int* rows, int n_rows, int hidden, const void* extra, const float* share,
                              cudaStream_t stream) {
    const bool aligned = (((uintptr_t)resid | (uintptr_t)delta | (uintptr_t)weight | (uintptr_t)out | (uintptr_t)extra) & 15) == 0;
    if (hidden % 8 == 0 && hidden <= 8192 && aligned) {
        MRUN_CHECK_CUDA(launch_kernel(add_rmsnorm_vec_kernel<TA, TD>, dim3(n_rows), dim3(256), 0, stream, resid,
                                   (const TD*)delta, weight, eps, (TA*)out, rows, hidden, (const TA*)extra, share), "add_rmsnorm");
        return 0;
    }
    const size_t smem = (size_t)hidden * sizeof(float);
    if (smem > 48 * 1024)
        MRUN_CHECK_CUDA(cudaFuncSetAttribute(add_rmsnorm_kernel<TA, TD>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             (int)smem), "add_rmsnorm");
    add_rmsnorm_kernel<TA, TD><<<n_rows, 256, smem, stream>>>(resid, (const TD*)delta, weight, eps, (TA*)out, rows,
                                                              hidden, (const TA*)extra, share);
    return 0;
}

// act_dtype: out's and extra's; delta_dtype: that or 32-bit.  extra and share (one factor a row) come together.
MRUN_API int mrun_add_rmsnorm(float* resid, const void* delta, int delta_dtype, const float* weight, float eps, void* out,
                              int act_dtype, const int* rows, int n_rows, int hidden, const void* extra,
                              const float* share, cudaStream_t stream) {
    MRUN_REQUIRE(n_rows >= 0 && hidden > 0, "add_rmsnorm: bad sizes rows=%d hidden=%d", n_rows, hidden);
    MRUN_REQUIRE((size_t)hidden * sizeof(float) <= 200 * 1024, "add_rmsnorm: hidden=%d exceeds the supported 51200",
                 hidden);
    MRUN_REQUIRE((extra == nullptr) == (share == nullptr), "add_rmsnorm: a second branch comes with its factors");
    MRUN_REQUIRE(delta_dtype == MRUN_F32 || delta_dtype == act_dtype, "add_rmsnorm: the branch is 32-bit or of the output's type");
    if (n_rows == 0) return 0;
    int rc;
    if (act_dtype == MRUN_F32)
        rc = launch_add_rmsnorm<float, float>(resid, delta, weight, eps, out, rows, n_rows, hidden, extra, share, stream);
    else if (act_dtype == MRUN_BF16 && delta_dtype == MRUN_F32)
        rc = launch_add_rmsnorm<__nv_bfloat16, float>(resid, delta, weight, eps, out, rows, n_rows, hidden, extra, share, stream);
    else if (act_dtype == MRUN_BF16)
        rc = launch_add_rmsnorm<__nv_bfloat16, __nv_bfloat16>(resid, delta, weight, eps, out, rows, n_rows, hidden, extra, share,
                                                              stream);
    else
        return mrun_set_error("add_rmsnorm: unknown dtype code %d", act_dtype);
    if (rc) return rc;
    MRUN_CHECK_LAUNCH("add_rmsnorm");
    return 0;
}

// ------------------------------------------------------------------------------------------
// y[t, :] += share[t] * x[t, :], the sum in 32-bit and rounded once to y's type: a branch that is a row
// itself with a factor (an identity expert) where no other kernel adds it.
// ------------------------------------------------------------------------------------------
template <typename TY, typename TX>
__global__ void add_scaled_rows_kernel(TY* __restrict__ y, const TX* __restrict__ x, const float* __restrict__ share,
                                       int width) {
    const float part = share[blockIdx.x];
    if (part == 0.f) return;
    const size_t row = (size_t)blockIdx.x * width;
    for (int c = threadIdx.x; c < width; c += blockDim.x) y[row + c] = from_float<TY>(fmaf(part, to_float(x[row + c]), to_float(y[row + c])));
}

MRUN_API int mrun_add_scaled_rows(void* y, int y_dtype, const void* x, int x_dtype, const float* share, int rows, int width,
                                  cudaStream_t stream) {
    MRUN_REQUIRE(rows >= 0 && width > 0 && share != nullptr, "add_scaled_rows: bad sizes rows=%d width=%d", rows, width);
    if (rows == 0) return 0;
    using bf16 = __nv_bfloat16;
    if (y_dtype == MRUN_F32 && x_dtype == MRUN_F32)
        add_scaled_rows_kernel<float, float><<<rows, 256, 0, stream>>>((float*)y, (const float*)x, share, width);
    else if (y_dtype == MRUN_F32 && x_dtype == MRUN_BF16)
        add_scaled_rows_kernel<float, bf16><<<rows, 256, 0, stream>>>((float*)y, (const bf16*)x, share, width);
    else if (y_dtype == MRUN_BF16 && x_dtype == MRUN_BF16)
        add_scaled_rows_kernel<bf16, bf16><<<rows, 256, 0, stream>>>((bf16*)y, (const bf16*)x, share, width);
    else
        return mrun_set_error("add_scaled_rows: no kernel for the dtype codes %d and %d", y_dtype, x_dtype);
    MRUN_CHECK_LAUNCH("add_scaled_rows");
    return 0;
}

// ------------------------------------------------------------------------------------------
// Rotation table: out[t, j] = (cos a, sin a), a = position[t] * inv_freq[j], the product and the
// functions in 64-bit, rounded once (the reference's explicit form computes the angle in
// 64-bit too, crates/mrun-engine/src/models/common.rs:264-270).  Both are multiplied by
// `magnitude` (1 for plain rotary positions; a scaled encoding may lengthen the rotated vector).
// A negative position (padding) gives (1, 0).
// ------------------------------------------------------------------------------------------
__global__ void rotary_table_kernel(const int* __restrict__ positions, const double* __restrict__ inv_freq,
                                    float2* __restrict__ out, int tokens, int half, double magnitude) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= tokens * half) return;
    const int t = i / half, j = i - t * half;
    const int p = positions[t];
    if (p < 0) {
        out[i] = make_float2(1.f, 0.f);
        return;
    }
    double s, c;
    sincos((double)p * inv_freq[j], &s, &c);
    out[i] = make_float2((float)(c * magnitude), (float)(s * magnitude));
}

MRUN_API int mrun_rotary_table(const int* positions, const double* inv_freq, float* out, int tokens,
                               int half, double magnitude, cudaStream_t stream) {
    MRUN_REQUIRE(tokens >= 0 && half > 0, "rotary_table: bad sizes tokens=%d half=%d", tokens, half);
    if (tokens == 0) return 0;
    const int n = tokens * half;
    rotary_table_kernel<<<(n + 255) / 256, 256, 0, stream>>>(positions, inv_freq, (float2*)out, tokens, half, magnitude);
    MRUN_CHECK_LAUNCH("rotary_table");
    return 0;
}

// ------------------------------------------------------------------------------------------
// Per-head RMSNorm of q and k, rotation of q and k, write of k and v into pages.
//   qkv: [tokens, (heads + 2 kv_heads) * head_dim], q heads first, then k heads, then v heads.
//   q is normed and rotated in place.  k (normed, rotated) and v (as is) go to
//   cache[page, kv_head, offset, :] with page * page_size + offset = slots[t]; a negative slot
//   skips the write (padding token, or a layer that only reads a cache).
// Order of operations: norm before rotation, v untouched
// (crates/mrun-engine/src/models/common.rs:183,194-198); pairing (j, j + rotary_dim/2)
// (crates/mrun-engine/src/models/common.rs:221,271-280).
// One warp per (token, head); the head's vector is staged in shared memory in 32-bit.
// ------------------------------------------------------------------------------------------
template <typename TA>
__global__ void qk_norm_rope_cache_kernel(TA* __restrict__ qkv, const float* __restrict__ q_weight,
                                          const float* __restrict__ k_weight, float eps,
                                          const float2* __restrict__ rot, int rotary_dim,
                                          const int* __restrict__ slots, TA* __restrict__ k_cache,
                                          TA* __restrict__ v_cache, int tokens, int heads, int kv_heads,
                                          int head_dim, int page_size) {
    extern __shared__ float vec_buf[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int per_token = heads + 2 * kv_heads;
    const long item = (long)blockIdx.x * (blockDim.x >> 5) + warp;
    if (item >= (long)tokens * per_token) return;
    const int t = (int)(item / per_token), slot_head = (int)(item - (long)t * per_token);
    float* vec = vec_buf + warp * head_dim;
    TA* src = qkv + ((size_t)t * per_token + slot_head) * head_dim;

    const bool is_q = slot_head < heads;
    const bool is_k = !is_q && slot_head < heads + kv_heads;
    const int kv_head = is_q ? 0 : (is_k ? slot_head - heads : slot_head - heads - kv_heads);
    const int slot = slots ? slots[t] : -1;
    if (!is_q && slot < 0) return;

    TA* dst;
    if (is_q) {
        dst = src;
    } else {
        const int page = slot / page_size, off = slot - page * page_size;
        TA* cache = is_k ? k_cache : v_cache;
        dst = cache + (((size_t)page * kv_heads + kv_head) * page_size + off) * head_dim;
    }

    if (!is_q && !is_k) {  // v: plain copy
        for (int e = lane; e < head_dim; e += 32) dst[e] = src[e];
        return;
    }

    float ss = 0.f;
    for (int e = lane; e < head_dim; e += 32) {
        const float v = to_float(src[e]);
        vec[e] = v;
        ss += v * v;
    }
    const float* weight = is_q ? q_weight : k_weight;
    if (weight) {
        ss = warp_sum(ss);
        const float inv = rsqrtf(ss / (float)head_dim + eps);
        __syncwarp();
        for (int e = lane; e < head_dim; e += 32) vec[e] = vec[e] * inv * weight[e];
    }
    __syncwarp();
    const int half = rotary_dim >> 1;
    if (rot) {
        const float2* cs = rot + (size_t)t * half;
        for (int j = lane; j < half; j += 32) {
            const float x1 = vec[j], x2 = vec[j + half];
            const float2 c = cs[j];
            dst[j] = from_float<TA>(x1 * c.x - x2 * c.y);
            dst[j + half] = from_float<TA>(x2 * c.x + x1 * c.y);
        }
        for (int e = rotary_dim + lane; e < head_dim; e += 32) dst[e] = from_float<TA>(vec[e]);
    } else {
        for (int e = lane; e < head_dim; e += 32) dst[e] = from_float<TA>(vec[e]);
    }
}

// The same for bfloat16 with a head of 64, 128 or 256 values rotated as a whole (or not at all):
// LANES = head_dim / 8 lanes share a head, eight values (16 bytes) a lane, so a row is read and
// written in whole 16-byte pieces; the sum of squares and the rotation's partner values (the lane
// LANES / 2 further along holds j + head_dim / 2) travel by shuffles.  A group of lanes takes
// QK_HEADS_PER_GROUP consecutive heads of one token, so the token's cosines and sines and the
// norm weights are read once for all of them.  The arithmetic is the scalar kernel's, value by value.
constexpr int QK_HEADS_PER_GROUP = 4;    // the fastest of 2, 4 and 8 heads a lane group on B200

template <int LANES>
__global__ void __launch_bounds__(256, 4)
qk_norm_rope_cache_vec_kernel(__nv_bfloat16* __restrict__ qkv, const float* __restrict__ q_weight,
                              const float* __restrict__ k_weight, float eps, const float2* __restrict__ rot,
                              const int* __restrict__ slots, __nv_bfloat16* __restrict__ k_cache,
                              __nv_bfloat16* __restrict__ v_cache, int tokens, int heads, int kv_heads,
                              int page_size) {
    constexpr int HEAD_DIM = LANES * 8, HALF = HEAD_DIM / 2;
    const int per_token = heads + 2 * kv_heads;
    const int groups_per_token = (per_token + QK_HEADS_PER_GROUP - 1) / QK_HEADS_PER_GROUP;
    const long group = ((long)blockIdx.x * blockDim.x + threadIdx.x) / LANES;
    const int part = threadIdx.x % LANES;                 // which eight values of a head
    // the lanes of a group leave together, so the shuffles below see all of them
    if (group >= (long)tokens * groups_per_token) return;
    const int t = (int)(group / groups_per_token);
    const int head0 = (int)(group - (long)t * groups_per_token) * QK_HEADS_PER_GROUP;
    const int head1 = min(per_token, head0 + QK_HEADS_PER_GROUP);
    const int slot = slots ? slots[t] : -1;
    const unsigned lane = threadIdx.x & 31;
    const unsigned mask = LANES == 32 ? 0xffffffffu : (((1u << LANES) - 1u) << (lane & ~(unsigned)(LANES - 1)));
    const bool upper = part >= LANES / 2;

    float cs[16];                                          // (cos, sin) of the lane's eight pairs
    if (rot && head0 < heads + kv_heads) {
        const float4* src = reinterpret_cast<const float4*>(rot + (size_t)t * HALF + (part % (LANES / 2)) * 8);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float4 c = src[i];
            cs[4 * i] = c.x; cs[4 * i + 1] = c.y; cs[4 * i + 2] = c.z; cs[4 * i + 3] = c.w;
        }
    }
    const __nv_bfloat16* row = qkv + (size_t)t * per_token * HEAD_DIM + part * 8;
    uint4 raw[QK_HEADS_PER_GROUP];
#pragma unroll
    for (int i = 0; i < QK_HEADS_PER_GROUP; ++i)
        if (head0 + i < head1) raw[i] = *reinterpret_cast<const uint4*>(row + (size_t)(head0 + i) * HEAD_DIM);

#pragma unroll
    for (int i = 0; i < QK_HEADS_PER_GROUP; ++i) {
        const int head = head0 + i;
        if (head >= head1) break;
        const bool is_q = head < heads;
        const bool is_k = !is_q && head < heads + kv_heads;
        if (!is_q && slot < 0) continue;
        __nv_bfloat16* dst = qkv + ((size_t)t * per_token + head) * HEAD_DIM + part * 8;
        if (!is_q) {
            const int kv_head = is_k ? head - heads : head - heads - kv_heads;
            const int page = slot / page_size, off = slot - page * page_size;
            dst = (is_k ? k_cache : v_cache) + (((size_t)page * kv_heads + kv_head) * page_size + off) * HEAD_DIM + part * 8;
        }
        if (!is_q && !is_k) {                              // v: plain copy
            *reinterpret_cast<uint4*>(dst) = raw[i];
            continue;
        }
        float v[8];
        {
            const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw[i]);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 f = __bfloat1622float2(pairs[e]);
                v[2 * e] = f.x; v[2 * e + 1] = f.y;
            }
        }
        const float* weight = is_q ? q_weight : k_weight;
        if (weight) {
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss += v[e] * v[e];
#pragma unroll
            for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(mask, ss, o);
            const float inv = rsqrtf(ss / (float)HEAD_DIM + eps);
            const float4 w0 = *reinterpret_cast<const float4*>(weight + part * 8);
            const float4 w1 = *reinterpret_cast<const float4*>(weight + part * 8 + 4);
            const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = v[e] * inv * w[e];
        }
        if (rot) {
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const float other = __shfl_xor_sync(mask, v[e], LANES / 2);
                // lower half: x1 cos - x2 sin; upper half: x2 cos + x1 sin
                v[e] = upper ? v[e] * cs[2 * e] + other * cs[2 * e + 1] : v[e] * cs[2 * e] - other * cs[2 * e + 1];
            }
        }
        uint4 packed;
        __nv_bfloat162* out = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
        for (int e = 0; e < 4; ++e) out[e] = __floats2bfloat162_rn(v[2 * e], v[2 * e + 1]);
        *reinterpret_cast<uint4*>(dst) = packed;
    }
}

template <int LANES>
cudaError_t launch_qk_vec(__nv_bfloat16* qkv, const float* q_weight, const float* k_weight, float eps, const float2* rot,
                          const int* slots, __nv_bfloat16* k_cache, __nv_bfloat16* v_cache, int tokens, int heads,
                          int kv_heads, int page_size, cudaStream_t stream) {
    const int per_token = heads + 2 * kv_heads;
    const long groups = (long)tokens * ((per_token + QK_HEADS_PER_GROUP - 1) / QK_HEADS_PER_GROUP);
    const long threads = groups * LANES;
    return launch_kernel(qk_norm_rope_cache_vec_kernel<LANES>, dim3((unsigned)((threads + 255) / 256)),
                      dim3(256), 0, stream, qkv, q_weight, k_weight, eps, rot, slots, k_cache, v_cache, tokens, heads,
                      kv_heads, page_size);
}

MRUN_API int mrun_qk_norm_rope_cache(void* qkv, int act_dtype, const float* q_weight, const float* k_weight,
                                     float eps, const float* rot, int rotary_dim, const int* slots,
                                     void* k_cache, void* v_cache, int tokens, int heads, int kv_heads,
                                     int head_dim, int page_size, cudaStream_t stream) {
    MRUN_REQUIRE(tokens >= 0 && heads > 0 && kv_heads > 0 && head_dim > 0 && page_size > 0,
                 "qk_norm_rope_cache: bad sizes");
    MRUN_REQUIRE(head_dim <= 1024, "qk_norm_rope_cache: head_dim=%d exceeds the supported 1024", head_dim);
    MRUN_REQUIRE(rotary_dim >= 0 && rotary_dim <= head_dim && rotary_dim % 2 == 0,
                 "qk_norm_rope_cache: rotary_dim=%d must be even and at most head_dim=%d", rotary_dim,
                 head_dim);
    MRUN_REQUIRE((q_weight == nullptr) == (k_weight == nullptr),
                 "qk_norm_rope_cache: q and k norm weights come together");
    MRUN_REQUIRE(slots == nullptr || (k_cache && v_cache), "qk_norm_rope_cache: slots without a cache");
    if (tokens == 0) return 0;
    const bool aligned = ((uintptr_t)qkv & 15) == 0 && ((uintptr_t)k_cache & 15) == 0 && ((uintptr_t)v_cache & 15) == 0 &&
                         ((uintptr_t)q_weight & 15) == 0 && ((uintptr_t)k_weight & 15) == 0 && ((uintptr_t)rot & 15) == 0;
    if (act_dtype == MRUN_BF16 && aligned && (rot == nullptr || rotary_dim == head_dim) &&
        (head_dim == 64 || head_dim == 128 || head_dim == 256)) {
        __nv_bfloat16* x = (__nv_bfloat16*)qkv;
        __nv_bfloat16 *kc = (__nv_bfloat16*)k_cache, *vc = (__nv_bfloat16*)v_cache;
        const float2* r = (const float2*)rot;
        cudaError_t err = head_dim == 64 ? launch_qk_vec<8>(x, q_weight, k_weight, eps, r, slots, kc, vc, tokens, heads, kv_heads, page_size, stream)
                        : head_dim == 128 ? launch_qk_vec<16>(x, q_weight, k_weight, eps, r, slots, kc, vc, tokens, heads, kv_heads, page_size, stream)
                                          : launch_qk_vec<32>(x, q_weight, k_weight, eps, r, slots, kc, vc, tokens, heads, kv_heads, page_size, stream);
        MRUN_CHECK_CUDA(err, "qk_norm_rope_cache");
        MRUN_CHECK_LAUNCH("qk_norm_rope_cache");
        return 0;
    }
    const int warps = 4;
    const long items = (long)tokens * (heads + 2 * kv_heads);
    const unsigned blocks = (unsigned)((items + warps - 1) / warps);
    const size_t smem = (size_t)warps * head_dim * sizeof(float);
    if (act_dtype == MRUN_F32)
        MRUN_CHECK_CUDA(launch_kernel(qk_norm_rope_cache_kernel<float>, dim3(blocks), dim3(warps * 32), smem, stream,
                                   (float*)qkv, q_weight, k_weight, eps, (const float2*)rot, rotary_dim, slots,
                                   (float*)k_cache, (float*)v_cache, tokens, heads, kv_heads, head_dim, page_size),
                        "qk_norm_rope_cache");
    else if (act_dtype == MRUN_BF16)
        MRUN_CHECK_CUDA(launch_kernel(qk_norm_rope_cache_kernel<__nv_bfloat16>, dim3(blocks), dim3(warps * 32), smem,
                                   stream, (__nv_bfloat16*)qkv, q_weight, k_weight, eps, (const float2*)rot,
                                   rotary_dim, slots, (__nv_bfloat16*)k_cache, (__nv_bfloat16*)v_cache, tokens, heads,
                                   kv_heads, head_dim, page_size),
                        "qk_norm_rope_cache");
    else
        return mrun_set_error("qk_norm_rope_cache: unknown dtype code %d", act_dtype);
    MRUN_CHECK_LAUNCH("qk_norm_rope_cache");
    return 0;
}

// ------------------------------------------------------------------------------------------
// RMS norm of q and of k over the whole projection (all heads of a token together, one weight per
// feature, eps inside the root), rotation of the first rotary_dim features of every q and k head,
// write of k and v into pages whose key and value sizes may differ.
//   x: row t at x + t * ld; the q heads ([heads, dim]) start at column q_off, the k heads
//   ([kv_heads, dim]) at k_off, the v heads ([kv_heads, vdim]) at v_off.  k_off < 0: the row has no
//   keys and values (a layer that reads another layer's pages) and only q is worked on.
//   q is normed and rotated in place.  k (normed, rotated) and v (as is) go to the pages at
//   slots[t]; a negative slot skips the write.  pairing: 0 = feature i with i + rotary_dim/2,
//   1 = feature 2i with 2i + 1; rot holds (cos, sin) per token and pair.
// One block a token; the token's q and k rows are staged in shared memory in 32-bit.
// ------------------------------------------------------------------------------------------
template <typename TA>
__global__ void __launch_bounds__(256)
proj_norm_rope_cache_kernel(TA* __restrict__ x, long ld, long q_off, long k_off, long v_off,
                            const float* __restrict__ q_weight, const float* __restrict__ k_weight, float eps,
                            const float2* __restrict__ rot, int rotary_dim, int pairing,
                            const int* __restrict__ slots, TA* __restrict__ k_cache, TA* __restrict__ v_cache,
                            int heads, int kv_heads, int dim, int vdim, int page_size) {
    extern __shared__ float staged[];         // heads * dim, then kv_heads * dim
    __shared__ float scratch[33];
    const int t = blockIdx.x, tid = threadIdx.x;
    TA* row = x + (size_t)t * ld;
    const int nq = heads * dim, nk = kv_heads * dim;
    const int slot = slots ? slots[t] : -1;
    const bool own = k_off >= 0 && slot >= 0;
    float* qv = staged;
    float* kv = staged + nq;

    float ss = 0.f;
    for (int e = tid; e < nq; e += blockDim.x) {
        const float v = to_float(row[q_off + e]);
        qv[e] = v;
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, scratch);
    if (q_weight) {
        const float inv = 1.f / sqrtf(ss / (float)nq + eps);
        for (int e = tid; e < nq; e += blockDim.x) qv[e] = qv[e] * inv * q_weight[e];
    }
    if (own) {
        float sk = 0.f;
        for (int e = tid; e < nk; e += blockDim.x) {
            const float v = to_float(row[k_off + e]);
            kv[e] = v;
            sk = fmaf(v, v, sk);
        }
        sk = block_sum(sk, scratch);
        if (k_weight) {
            const float inv = 1.f / sqrtf(sk / (float)nk + eps);
            for (int e = tid; e < nk; e += blockDim.x) kv[e] = kv[e] * inv * k_weight[e];
        }
    }
    __syncthreads();

    const int half = rotary_dim >> 1;
    const float2* cs = rot ? rot + (size_t)t * half : nullptr;
    auto rotated = [&](const float* head, int e) -> float {
        if (!cs || e >= rotary_dim) return head[e];
        int pair, partner;
        bool first;
        if (pairing) { pair = e >> 1; partner = e ^ 1; first = (e & 1) == 0; }
        else { first = e < half; pair = first ? e : e - half; partner = first ? e + half : e - half; }
        const float2 c = cs[pair];
        return first ? head[e] * c.x - head[partner] * c.y : head[e] * c.x + head[partner] * c.y;
    };
    for (int i = tid; i < nq; i += blockDim.x) {
        const int h = i / dim, e = i - h * dim;
        row[q_off + i] = from_float<TA>(rotated(qv + h * dim, e));
    }
    if (!own) return;
    const int page = slot / page_size, off = slot - page * page_size;
    for (int i = tid; i < nk; i += blockDim.x) {
        const int g = i / dim, e = i - g * dim;
        k_cache[(((size_t)page * kv_heads + g) * page_size + off) * dim + e] = from_float<TA>(rotated(kv + g * dim, e));
    }
    for (int i = tid; i < kv_heads * vdim; i += blockDim.x) {
        const int g = i / vdim, e = i - g * vdim;
        v_cache[(((size_t)page * kv_heads + g) * page_size + off) * vdim + e] = row[v_off + i];
    }
}

MRUN_API int mrun_proj_norm_rope_cache(void* x, long ld, long q_off, long k_off, long v_off, int act_dtype,
                                       const float* q_weight, const float* k_weight, float eps, const float* rot,
                                       int rotary_dim, int pairing, const int* slots, void* k_cache, void* v_cache,
                                       int tokens, int heads, int kv_heads, int dim, int vdim, int page_size,
                                       cudaStream_t stream) {
    MRUN_REQUIRE(tokens >= 0 && heads > 0 && kv_heads > 0 && dim > 0 && vdim > 0 && page_size > 0,
                 "proj_norm_rope_cache: bad sizes");
    MRUN_REQUIRE(rotary_dim >= 0 && rotary_dim <= dim && rotary_dim % 2 == 0,
                 "proj_norm_rope_cache: rotary_dim=%d must be even and at most dim=%d", rotary_dim, dim);
    MRUN_REQUIRE(q_off >= 0 && (k_off < 0 || v_off >= 0), "proj_norm_rope_cache: bad column offsets");
    MRUN_REQUIRE(k_off < 0 || slots == nullptr || (k_cache && v_cache), "proj_norm_rope_cache: slots without a cache");
    const size_t smem = (size_t)(heads + kv_heads) * dim * sizeof(float);
    MRUN_REQUIRE(smem <= 200 * 1024, "proj_norm_rope_cache: %d q and k features a token exceed the supported 51200",
                 (heads + kv_heads) * dim);
    if (tokens == 0) return 0;
    const float2* cs = rotary_dim ? (const float2*)rot : nullptr;
    if (act_dtype == MRUN_F32) {
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(proj_norm_rope_cache_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        proj_norm_rope_cache_kernel<float><<<tokens, 256, smem, stream>>>(
            (float*)x, ld, q_off, k_off, v_off, q_weight, k_weight, eps, cs, rotary_dim, pairing, slots, (float*)k_cache,
            (float*)v_cache, heads, kv_heads, dim, vdim, page_size);
    } else if (act_dtype == MRUN_BF16) {
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(proj_norm_rope_cache_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 (int)smem);
        proj_norm_rope_cache_kernel<__nv_bfloat16><<<tokens, 256, smem, stream>>>(
            (__nv_bfloat16*)x, ld, q_off, k_off, v_off, q_weight, k_weight, eps, cs, rotary_dim, pairing, slots,
            (__nv_bfloat16*)k_cache, (__nv_bfloat16*)v_cache, heads, kv_heads, dim, vdim, page_size);
    } else {
        return mrun_set_error("proj_norm_rope_cache: unknown dtype code %d", act_dtype);
    }
    MRUN_CHECK_LAUNCH("proj_norm_rope_cache");
    return 0;
}

// ------------------------------------------------------------------------------------------
// Gated activation: out[t, i] = act(gate_i) * up_i in 32-bit; act by code: SiLU
// (z * sigmoid(z), crates/mrun-engine/src/models/activations.rs:46-59) or tanh-GELU.
// Layout of gate_up[t, :]: block == 0: all gates, then all ups (gate_i at i, up_i at inter + i).
// block == 8: runs of eight gates followed by the eight ups of the same outputs
// (gate_i at 16 (i / 8) + i % 8, up_i eight further), the row order the decode GEMM's fused
// epilogue wants of the stacked weight.
// ------------------------------------------------------------------------------------------
template <typename TA>
__global__ void swiglu_kernel(const TA* __restrict__ gate_up, TA* __restrict__ out, long total, int inter,
                              int block, int act) {
    const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const long t = i / inter;
    const int c = (int)(i - t * inter);
    const long gi = block ? t * 2 * inter + 2 * (c & ~7) + (c & 7) : t * 2 * inter + c;
    const long ui = block ? gi + 8 : gi + inter;
    const float g = to_float(gate_up[gi]);
    const float u = to_float(gate_up[ui]);
    out[i] = from_float<TA>(mrun::gated_mul<sizeof(TA) == 4>(act, g, u));
}

// Eight outputs per thread with 16-byte loads and stores, for widths that are a multiple of 8.
// One group a thread: with two or four groups in flight per thread the kernel was slower
// (by 10 to 50 per cent at 2,048 x 12,288 outputs).
template <typename TA>
__global__ void __launch_bounds__(256)
swiglu_vec_kernel(const TA* __restrict__ gate_up, TA* __restrict__ out, long total8, int inter, int block, int act) {
    const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total8) return;
    const int per_row = inter >> 3;
    const long t = i / per_row;
    const int c = (int)(i - t * per_row) << 3;
    const TA* g_ptr = gate_up + t * 2 * inter + (block ? 2 * c : c);
    const TA* u_ptr = block ? g_ptr + 8 : g_ptr + inter;
    float g[8], u[8], y[8];
    Vec8<TA>::load(g_ptr, g);
    Vec8<TA>::load(u_ptr, u);
#pragma unroll
    for (int e = 0; e < 8; ++e) y[e] = mrun::gated_mul<sizeof(TA) == 4>(act, g[e], u[e]);
    Vec8<TA>::store(out + t * inter + c, y);
}

MRUN_API int mrun_swiglu(const void* gate_up, void* out, int act_dtype, int tokens, int inter, int block,
                         int act, cudaStream_t stream) {
    MRUN_REQUIRE_GATE(act, "swiglu");
    MRUN_REQUIRE(tokens >= 0 && inter > 0, "swiglu: bad sizes tokens=%d inter=%d", tokens, inter);
    MRUN_REQUIRE(block == 0 || (block == 8 && inter % 8 == 0),
                 "swiglu: the interleaved layout has runs of 8 and needs inter=%d to be a multiple of 8", inter);
    if (tokens == 0) return 0;
    const long total = (long)tokens * inter;
    const bool aligned = (((uintptr_t)gate_up | (uintptr_t)out) & 15) == 0;
    if (inter % 8 == 0 && aligned && (act_dtype == MRUN_F32 || act_dtype == MRUN_BF16)) {
        const long total8 = total / 8;
        const unsigned vblocks = (unsigned)((total8 + 255) / 256);
        if (act_dtype == MRUN_F32)
            swiglu_vec_kernel<float><<<vblocks, 256, 0, stream>>>((const float*)gate_up, (float*)out, total8, inter,
                                                                block, act);
        else
            swiglu_vec_kernel<__nv_bfloat16><<<vblocks, 256, 0, stream>>>(
                (const __nv_bfloat16*)gate_up, (__nv_bfloat16*)out, total8, inter, block, act);
        MRUN_CHECK_LAUNCH("swiglu");
        return 0;
    }
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (act_dtype == MRUN_F32)
        swiglu_kernel<float><<<blocks, 256, 0, stream>>>((const float*)gate_up, (float*)out, total, inter, block, act);
    else if (act_dtype == MRUN_BF16)
        swiglu_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)gate_up,
                                                                 (__nv_bfloat16*)out, total, inter, block, act);
    else
        return mrun_set_error("swiglu: unknown dtype code %d", act_dtype);
    MRUN_CHECK_LAUNCH("swiglu");
    return 0;
}

// ------------------------------------------------------------------------------------------
// Bias of a linear layer: y[t, n] += bias[n], the sum in 32-bit and rounded once to y's type
// (crates/mrun-engine/src/load.rs:302-305 adds an optional bias after the product).
// ------------------------------------------------------------------------------------------
template <typename TA>
__global__ void add_bias_kernel(TA* __restrict__ y, const float* __restrict__ bias, long total, int n) {
    const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    y[i] = from_float<TA>(to_float(y[i]) + bias[(int)(i % n)]);
}

MRUN_API int mrun_add_bias(void* y, int act_dtype, const float* bias, int tokens, int n, cudaStream_t stream) {
    MRUN_REQUIRE(tokens >= 0 && n > 0, "add_bias: bad sizes tokens=%d n=%d", tokens, n);
    if (tokens == 0) return 0;
    const long total = (long)tokens * n;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (act_dtype == MRUN_F32)
        add_bias_kernel<float><<<blocks, 256, 0, stream>>>((float*)y, bias, total, n);
    else if (act_dtype == MRUN_BF16)
        add_bias_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((__nv_bfloat16*)y, bias, total, n);
    else
        return mrun_set_error("add_bias: unknown dtype code %d", act_dtype);
    MRUN_CHECK_LAUNCH("add_bias");
    return 0;
}

// ------------------------------------------------------------------------------------------
// Scatter of 32-bit integers: dst[index[i]] = value[i].  Brings the block tables on the device up
// to date with the pages the host handed out or took back since the last step.
// ------------------------------------------------------------------------------------------
__global__ void scatter_i32_kernel(int* __restrict__ dst, const int* __restrict__ index,
                                   const int* __restrict__ value, int n, long dst_size) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const long at = index[i];
    if (at >= 0 && at < dst_size) dst[at] = value[i];
}

MRUN_API int mrun_scatter_i32(int* dst, const int* index, const int* value, int n, long dst_size,
                              cudaStream_t stream) {
    MRUN_REQUIRE(n >= 0 && dst_size >= 0, "scatter_i32: bad sizes n=%d dst_size=%ld", n, dst_size);
    if (n == 0) return 0;
    scatter_i32_kernel<<<(n + 255) / 256, 256, 0, stream>>>(dst, index, value, n, dst_size);
    MRUN_CHECK_LAUNCH("scatter_i32");
    return 0;
}

// ------------------------------------------------------------------------------------------
// Token feedback: ids[r] = previous[source[r]] where source[r] >= 0.  Lets a decode step take the
// tokens the step before it sampled straight from the device, before the host has read them
// (the reference feeds a sampled token before reading it back too,
// crates/mrun-engine/src/nuvec_engine.rs:1489-1500).
// ------------------------------------------------------------------------------------------
__global__ void select_tokens_kernel(int* __restrict__ ids, const int* __restrict__ previous,
                                     const int* __restrict__ source, int rows, int previous_rows) {
    const int r = blockIdx.x * blockDim.x + threadIdx.x;
    if (r >= rows) return;
    const int s = source[r];
    if (s >= 0 && s < previous_rows) ids[r] = previous[s];
}

MRUN_API int mrun_select_tokens(int* ids, const int* previous, const int* source, int rows, int previous_rows,
                                cudaStream_t stream) {
    MRUN_REQUIRE(rows >= 0 && previous_rows >= 0, "select_tokens: bad sizes rows=%d previous=%d", rows, previous_rows);
    if (rows == 0) return 0;
    select_tokens_kernel<<<(rows + 255) / 256, 256, 0, stream>>>(ids, previous, source, rows, previous_rows);
    MRUN_CHECK_LAUNCH("select_tokens");
    return 0;
}


// ------------------------------------------------------------------------------------------
// A gate per head, in place: y[t, h, :] *= sigmoid(gate[t, h]).  `gate` rows are `ldg` elements
// apart (a column slice of a wider product); the sigmoid is 32-bit.  For attention kernels that
// write finished heads and know nothing of a gate.
// ------------------------------------------------------------------------------------------
template <typename TA>
__global__ void head_gate_kernel(TA* __restrict__ y, const TA* __restrict__ gate, long ldg, long total, int heads, int n) {
    const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const long pair = i / n;                 // (token, head)
    const long t = pair / heads;
    const float g = to_float(gate[t * ldg + (pair - t * heads)]);
    y[i] = from_float<TA>(to_float(y[i]) / (1.f + expf(-g)));
}

// The same for bfloat16 heads whose size is a multiple of 8: a thread takes 8 features (16 bytes)
// of one head.
__global__ void head_gate_vec_kernel(uint4* __restrict__ y, const __nv_bfloat16* __restrict__ gate, long ldg, long total8,
                                     int heads, int n8) {
    const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total8) return;
    const long pair = i / n8;
    const long t = pair / heads;
    const float s = 1.f / (1.f + expf(-__bfloat162float(gate[t * ldg + (pair - t * heads)])));
    uint4 v = y[i];
    __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const float2 f = __bfloat1622float2(p[j]);
        p[j] = __floats2bfloat162_rn(f.x * s, f.y * s);
    }
    y[i] = v;
}

MRUN_API int mrun_head_gate(void* y, const void* gate, long ldg, int act_dtype, int tokens, int heads, int n,
                            cudaStream_t stream) {
    MRUN_REQUIRE(tokens >= 0 && heads > 0 && n > 0 && ldg >= heads, "head_gate: bad sizes tokens=%d heads=%d n=%d ldg=%ld",
                 tokens, heads, n, ldg);
    if (tokens == 0) return 0;
    const long total = (long)tokens * heads * n;
    if (act_dtype == MRUN_BF16 && n % 8 == 0 && ((uintptr_t)y & 15) == 0) {
        const long total8 = total / 8;
        head_gate_vec_kernel<<<(unsigned)((total8 + 255) / 256), 256, 0, stream>>>((uint4*)y, (const __nv_bfloat16*)gate, ldg,
                                                                                  total8, heads, n / 8);
        MRUN_CHECK_LAUNCH("head_gate");
        return 0;
    }
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (act_dtype == MRUN_F32)
        head_gate_kernel<float><<<blocks, 256, 0, stream>>>((float*)y, (const float*)gate, ldg, total, heads, n);
    else if (act_dtype == MRUN_BF16)
        head_gate_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((__nv_bfloat16*)y, (const __nv_bfloat16*)gate, ldg, total,
                                                                    heads, n);
    else
        return mrun_set_error("head_gate: unknown dtype code %d", act_dtype);
    MRUN_CHECK_LAUNCH("head_gate");
    return 0;
}

// ------------------------------------------------------------------------------------------
// Per-head RMS norm of q and k (one weight of `dim` entries that the heads share, eps inside the
// root), rotation of the first `rotary_dim` features of every head in either pairing, k and v into
// the pages, for rows whose q, k and v heads start at columns of their own (q_off, k_off, v_off)
// and whose keys (`dim` a head) and values (`vdim` a head) may differ in size.
//   v_off < 0: the layer has no value projection and the values are the keys as they were
//   projected, before the norm and the rotation (vdim = dim).
//   HeadExtras: biases of the projections, added before anything else; values kept for a later layer
//   of the step, and values blended with those an earlier layer kept.
// q is worked on in place; a negative slot skips the page writes.  One warp per (token, q or k
// or v head); the head's vector is staged in shared memory in 32-bit.
// ------------------------------------------------------------------------------------------
struct HeadExtras {
    const float* bias;          // [q heads | k heads | v heads] or null
    const void* first;          // row t's values of an earlier layer at first + t * ld_first (the activation type), or null
    long ld_first;
    float share;                // v <- (1 - share) * v + share * first
    void* keep;                 // gets v (with its bias, before the blend), row t at keep + t * ld_keep; or null
    long ld_keep;
};

// Eight (or fewer) features of a value head from feature e of the token's value row on.
template <typename TA, int N>
__device__ __forceinline__ void extend_values(const HeadExtras& x, const float* vbias, int t, int e, float (&v)[N]) {
    if (vbias)
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] += vbias[e + i];
    if (x.keep)
#pragma unroll
        for (int i = 0; i < N; ++i) ((TA*)x.keep)[(size_t)t * x.ld_keep + e + i] = from_float<TA>(v[i]);
    if (x.first)
#pragma unroll
        for (int i = 0; i < N; ++i)
            v[i] = (1.f - x.share) * v[i] + x.share * to_float(((const TA*)x.first)[(size_t)t * x.ld_first + e + i]);
}

template <typename TA>
__global__ void head_norm_rope_cache_kernel(TA* __restrict__ x, long ld, long q_off, long k_off, long v_off,
                                            const float* __restrict__ q_weight, const float* __restrict__ k_weight,
                                            float eps, const float2* __restrict__ rot, int rotary_dim, int interleaved,
                                            const int* __restrict__ slots, TA* __restrict__ k_cache,
                                            TA* __restrict__ v_cache, int tokens, int heads, int kv_heads, int dim,
                                            int vdim, int page_size, const HeadExtras extras) {
    extern __shared__ float vec_buf[];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int per_token = heads + (v_off >= 0 ? 2 : 1) * kv_heads;
    const long item = (long)blockIdx.x * (blockDim.x >> 5) + warp;
    if (item >= (long)tokens * per_token) return;
    const int t = (int)(item / per_token), slot_head = (int)(item - (long)t * per_token);
    const bool is_q = slot_head < heads;
    const bool is_k = !is_q && slot_head < heads + kv_heads;
    const int slot = slots ? slots[t] : -1;
    if (!is_q && slot < 0 && (is_k || !extras.keep)) return;
    const int page = slot >= 0 ? slot / page_size : 0, off = slot >= 0 ? slot - page * page_size : 0;
    TA* row = x + (size_t)t * ld;
    if (!is_q && !is_k) {       // a value head of a projection of its own
        const int g = slot_head - heads - kv_heads;
        const TA* src = row + v_off + (size_t)g * vdim;
        TA* dst = slot < 0 ? nullptr : v_cache + (((size_t)page * kv_heads + g) * page_size + off) * vdim;
        const float* vbias = extras.bias ? extras.bias + (size_t)(heads + kv_heads) * dim : nullptr;
        for (int e = lane; e < vdim; e += 32) {
            float v[1] = {to_float(src[e])};
            extend_values<TA, 1>(extras, vbias, t, g * vdim + e, v);
            if (dst) dst[e] = from_float<TA>(v[0]);
        }
        return;
    }
    const int g = is_q ? slot_head : slot_head - heads;
    TA* src = row + (is_q ? q_off : k_off) + (size_t)g * dim;
    TA* dst = is_q ? src : k_cache + (((size_t)page * kv_heads + g) * page_size + off) * dim;
    float* vec = vec_buf + warp * dim;
    const float* bias = extras.bias ? extras.bias + (size_t)slot_head * dim : nullptr;
    float ss = 0.f;
    for (int e = lane; e < dim; e += 32) {
        const float v = to_float(src[e]) + (bias ? bias[e] : 0.f);
        vec[e] = v;
        ss += v * v;
    }
    if (is_k && v_off < 0) {    // the values are the keys as projected
        TA* vdst = v_cache + (((size_t)page * kv_heads + g) * page_size + off) * vdim;
        for (int e = lane; e < dim; e += 32) vdst[e] = from_float<TA>(vec[e]);
    }
    const float* weight = is_q ? q_weight : k_weight;
    if (weight) {
        ss = warp_sum(ss);
        const float inv = rsqrtf(ss / (float)dim + eps);
        __syncwarp();
        for (int e = lane; e < dim; e += 32) vec[e] = vec[e] * inv * weight[e];
    }
    __syncwarp();
    const int half = rotary_dim >> 1;
    if (rot && half > 0) {
        const float2* cs = rot + (size_t)t * half;
        for (int j = lane; j < half; j += 32) {
            const int a = interleaved ? 2 * j : j, b = interleaved ? 2 * j + 1 : j + half;
            const float x1 = vec[a], x2 = vec[b];
            const float2 c = cs[j];
            dst[a] = from_float<TA>(x1 * c.x - x2 * c.y);
            dst[b] = from_float<TA>(x2 * c.x + x1 * c.y);
        }
        for (int e = rotary_dim + lane; e < dim; e += 32) dst[e] = from_float<TA>(vec[e]);
    } else {
        for (int e = lane; e < dim; e += 32) dst[e] = from_float<TA>(vec[e]);
    }
}

// The same for bfloat16 heads of 16, 32, 64, 128 or 256 features with values of a multiple of 8,
// half-split pairs and a rotating part that is a multiple of 16 features (or none): LANES = dim / 8
// lanes share a head, eight values (16 bytes) a lane, so a row is read and written in whole 16-byte
// pieces; the sum of squares and the rotation's partner values (the lane rotary_dim / 16 further
// along holds j + rotary_dim / 2) travel by shuffles.  The arithmetic is the scalar kernel's, value
// by value.
template <int LANES>
__global__ void __launch_bounds__(128)
head_norm_rope_cache_vec_kernel(__nv_bfloat16* __restrict__ x, long ld, long q_off, long k_off, long v_off,
                                const float* __restrict__ q_weight, const float* __restrict__ k_weight, float eps,
                                const float2* __restrict__ rot, int rotary_dim, const int* __restrict__ slots,
                                __nv_bfloat16* __restrict__ k_cache, __nv_bfloat16* __restrict__ v_cache, int tokens,
                                int heads, int kv_heads, int vdim, int page_size, const HeadExtras extras) {
    constexpr int dim = LANES * 8;
    const int sub = threadIdx.x % LANES;                       // this lane's place in its head
    const int per_token = heads + (v_off >= 0 ? 2 : 1) * kv_heads;
    const long item = ((long)blockIdx.x * blockDim.x + threadIdx.x) / LANES;
    // lanes of a group leave together: the shuffles below name the group's lanes only
    const unsigned lane = threadIdx.x & 31;
    const unsigned group_mask = LANES == 32 ? 0xffffffffu : (((1u << LANES) - 1u) << (lane / LANES * LANES));
    if (item >= (long)tokens * per_token) return;
    const int t = (int)(item / per_token), slot_head = (int)(item - (long)t * per_token);
    const bool is_q = slot_head < heads;
    const bool is_k = !is_q && slot_head < heads + kv_heads;
    const int slot = slots ? slots[t] : -1;
    if (!is_q && slot < 0 && (is_k || !extras.keep)) return;
    const int page = slot >= 0 ? slot / page_size : 0, off = slot >= 0 ? slot - page * page_size : 0;
    __nv_bfloat16* row = x + (size_t)t * ld;
    if (!is_q && !is_k) {       // a value head of a projection of its own
        const int g = slot_head - heads - kv_heads;
        const __nv_bfloat16* src = row + v_off + (size_t)g * vdim;
        __nv_bfloat16* dst = slot < 0 ? nullptr : v_cache + (((size_t)page * kv_heads + g) * page_size + off) * vdim;
        const float* vbias = extras.bias ? extras.bias + (size_t)(heads + kv_heads) * dim : nullptr;
        for (int c = sub; c < (vdim >> 3); c += LANES) {
            if (vbias || extras.keep || extras.first) {
                float v[8];
                Vec8<__nv_bfloat16>::load(src + c * 8, v);
                extend_values<__nv_bfloat16, 8>(extras, vbias, t, g * vdim + c * 8, v);
                if (dst) Vec8<__nv_bfloat16>::store(dst + c * 8, v);
            } else {
                reinterpret_cast<uint4*>(dst)[c] = reinterpret_cast<const uint4*>(src)[c];
            }
        }
        return;
    }
    const int g = is_q ? slot_head : slot_head - heads;
    __nv_bfloat16* src = row + (is_q ? q_off : k_off) + (size_t)g * dim;
    __nv_bfloat16* dst = is_q ? src : k_cache + (((size_t)page * kv_heads + g) * page_size + off) * dim;
    const uint4 raw = reinterpret_cast<const uint4*>(src)[sub];
    float v[8];
    {
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(h[i]);
            v[2 * i] = f.x; v[2 * i + 1] = f.y;
        }
    }
    if (extras.bias) {
        float b[8];
        Vec8<float>::load(extras.bias + (size_t)slot_head * dim + sub * 8, b);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] += b[i];
    }
    if (is_k && v_off < 0)      // the values are the keys as projected
        Vec8<__nv_bfloat16>::store(v_cache + (((size_t)page * kv_heads + g) * page_size + off) * dim + sub * 8, v);
    const float* weight = is_q ? q_weight : k_weight;
    if (weight) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) ss += v[i] * v[i];
#pragma unroll
        for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(group_mask, ss, o);
        const float inv = rsqrtf(ss / (float)dim + eps);
        float w[8];
        Vec8<float>::load(weight + sub * 8, w);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = v[i] * inv * w[i];
    }
    if (rot && rotary_dim > 0) {
        const int hop = rotary_dim / 16;                       // lanes between a feature and its partner
        const bool first = sub < hop, second = !first && sub < 2 * hop;
        // every lane of the group takes part in the shuffles; lanes beyond the rotating part keep their values
        const int partner = first ? sub + hop : (second ? sub - hop : sub);
        float other[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) other[i] = __shfl_sync(group_mask, v[i], (lane / LANES) * LANES + partner);
        if (first || second) {
            const float2* cs = rot + (size_t)t * (rotary_dim >> 1) + (first ? sub : sub - hop) * 8;
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float2 c = cs[i];
                v[i] = first ? v[i] * c.x - other[i] * c.y : v[i] * c.x + other[i] * c.y;
            }
        }
    }
    Vec8<__nv_bfloat16>::store(dst + sub * 8, v);
}

template <int LANES>
static void launch_head_norm_rope_cache_vec(void* x, long ld, long q_off, long k_off, long v_off, const float* q_weight,
                                            const float* k_weight, float eps, const float* rot, int rotary_dim,
                                            const int* slots, void* k_cache, void* v_cache, int tokens, int heads,
                                            int kv_heads, int vdim, int page_size, const HeadExtras& extras,
                                            cudaStream_t stream) {
    const long items = (long)tokens * (heads + (v_off >= 0 ? 2 : 1) * kv_heads);
    const long threads = items * LANES;
    head_norm_rope_cache_vec_kernel<LANES><<<(unsigned)((threads + 127) / 128), 128, 0, stream>>>(
        (__nv_bfloat16*)x, ld, q_off, k_off, v_off, q_weight, k_weight, eps, (const float2*)rot, rotary_dim, slots,
        (__nv_bfloat16*)k_cache, (__nv_bfloat16*)v_cache, tokens, heads, kv_heads, vdim, page_size, extras);
}

MRUN_API int mrun_head_norm_rope_cache(void* x, long ld, long q_off, long k_off, long v_off, int act_dtype,
                                       const float* q_weight, const float* k_weight, float eps, const float* rot,
                                       int rotary_dim, int pairing, const int* slots, void* k_cache, void* v_cache,
                                       int tokens, int heads, int kv_heads, int dim, int vdim, int page_size,
                                       const float* bias, const void* first, long ld_first, float share, void* keep,
                                       long ld_keep, cudaStream_t stream) {
    MRUN_REQUIRE(tokens >= 0 && heads > 0 && kv_heads > 0 && dim > 0 && vdim > 0 && page_size > 0,
                 "head_norm_rope_cache: bad sizes tokens=%d heads=%d kv_heads=%d dim=%d vdim=%d page_size=%d", tokens,
                 heads, kv_heads, dim, vdim, page_size);
    MRUN_REQUIRE(rotary_dim >= 0 && rotary_dim % 2 == 0 && rotary_dim <= dim,
                 "head_norm_rope_cache: rotary_dim=%d must be even and at most dim=%d", rotary_dim, dim);
    MRUN_REQUIRE(pairing == 0 || pairing == 1, "head_norm_rope_cache: unknown pairing code %d", pairing);
    MRUN_REQUIRE(v_off >= 0 || vdim == dim, "head_norm_rope_cache: values that are the keys have the keys' size (%d), not %d",
                 dim, vdim);
    MRUN_REQUIRE(q_off >= 0 && k_off >= 0, "head_norm_rope_cache: negative column of q or k");
    MRUN_REQUIRE(v_off >= 0 || (first == nullptr && keep == nullptr),
                 "head_norm_rope_cache: values that are the keys are neither kept nor blended");
    MRUN_REQUIRE((first == nullptr || ld_first >= (long)kv_heads * vdim) && (keep == nullptr || ld_keep >= (long)kv_heads * vdim),
                 "head_norm_rope_cache: the kept values' rows do not hold %d features", kv_heads * vdim);
    const HeadExtras extras = {bias, first, ld_first, share, keep, ld_keep};
    MRUN_REQUIRE((size_t)dim * sizeof(float) * 4 <= 48 * 1024, "head_norm_rope_cache: dim=%d exceeds the supported 3072", dim);
    if (tokens == 0) return 0;
    const int warps = 4;
    const long items = (long)tokens * (heads + (v_off >= 0 ? 2 : 1) * kv_heads);
    const unsigned blocks = (unsigned)((items + warps - 1) / warps);
    const size_t smem = (size_t)warps * dim * sizeof(float);
    if (slots == nullptr) k_cache = v_cache = nullptr;
    const bool aligned = ((((uintptr_t)x) | ((uintptr_t)k_cache) | ((uintptr_t)v_cache) | ((uintptr_t)q_weight) |
                           ((uintptr_t)k_weight) | ((uintptr_t)bias)) & 15) == 0 &&
                         ld % 8 == 0 && q_off % 8 == 0 && k_off % 8 == 0 && (v_off < 0 || v_off % 8 == 0);
    if (act_dtype == MRUN_BF16 && aligned && vdim % 8 == 0 && (v_off >= 0 || vdim == dim) && pairing == 0 && rotary_dim % 16 == 0 &&
        (dim == 16 || dim == 32 || dim == 64 || dim == 128 || dim == 256)) {
#define MRUN_HEAD_VEC(L)                                                                                              \
    launch_head_norm_rope_cache_vec<L>(x, ld, q_off, k_off, v_off, q_weight, k_weight, eps, rot, rot ? rotary_dim : 0, \
                                       slots, k_cache, v_cache, tokens, heads, kv_heads, vdim, page_size, extras, stream)
        switch (dim) {
            case 16: MRUN_HEAD_VEC(2); break;
            case 32: MRUN_HEAD_VEC(4); break;
            case 64: MRUN_HEAD_VEC(8); break;
            case 128: MRUN_HEAD_VEC(16); break;
            default: MRUN_HEAD_VEC(32); break;
        }
#undef MRUN_HEAD_VEC
        MRUN_CHECK_LAUNCH("head_norm_rope_cache");
        return 0;
    }
    if (act_dtype == MRUN_F32)
        head_norm_rope_cache_kernel<float><<<blocks, warps * 32, smem, stream>>>(
            (float*)x, ld, q_off, k_off, v_off, q_weight, k_weight, eps, (const float2*)rot, rotary_dim, pairing, slots,
            (float*)k_cache, (float*)v_cache, tokens, heads, kv_heads, dim, vdim, page_size, extras);
    else if (act_dtype == MRUN_BF16)
        head_norm_rope_cache_kernel<__nv_bfloat16><<<blocks, warps * 32, smem, stream>>>(
            (__nv_bfloat16*)x, ld, q_off, k_off, v_off, q_weight, k_weight, eps, (const float2*)rot, rotary_dim, pairing,
            slots, (__nv_bfloat16*)k_cache, (__nv_bfloat16*)v_cache, tokens, heads, kv_heads, dim, vdim, page_size, extras);
    else
        return mrun_set_error("head_norm_rope_cache: unknown dtype code %d", act_dtype);
    MRUN_CHECK_LAUNCH("head_norm_rope_cache");
    return 0;
}

// ------------------------------------------------------------------------------------------
// out[i] = act(x[i]) in 32-bit, a function of one argument (MRUN_ACT_*); x and out may differ in type.
// ------------------------------------------------------------------------------------------
template <typename TX, typename TA>
__global__ void __launch_bounds__(256)
plain_act_kernel(const TX* __restrict__ x, TA* __restrict__ out, long n, int act) {
    const long i = (long)blockIdx.x * 256 + threadIdx.x;
    if (i < n) out[i] = from_float<TA>(plain_act(act, to_float(x[i])));
}

MRUN_API int mrun_plain_act(const void* x, int x_dtype, void* out, int out_dtype, long n, int act, cudaStream_t stream) {
    MRUN_REQUIRE(n >= 0 && (act == MRUN_ACT_RELU2 || act == MRUN_ACT_TANH), "plain_act: n=%ld, activation code %d", n, act);
    MRUN_REQUIRE(x_dtype == MRUN_F32 || x_dtype == MRUN_BF16, "plain_act: unknown dtype code %d", x_dtype);
    MRUN_REQUIRE(out_dtype == MRUN_F32 || out_dtype == MRUN_BF16, "plain_act: unknown dtype code %d", out_dtype);
    if (n == 0) return 0;
    const unsigned blocks = (unsigned)((n + 255) / 256);
    if (x_dtype == MRUN_F32 && out_dtype == MRUN_F32)
        plain_act_kernel<float, float><<<blocks, 256, 0, stream>>>((const float*)x, (float*)out, n, act);
    else if (x_dtype == MRUN_F32)
        plain_act_kernel<float, __nv_bfloat16><<<blocks, 256, 0, stream>>>((const float*)x, (__nv_bfloat16*)out, n, act);
    else if (out_dtype == MRUN_F32)
        plain_act_kernel<__nv_bfloat16, float><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)x, (float*)out, n, act);
    else
        plain_act_kernel<__nv_bfloat16, __nv_bfloat16><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)x,
                                                                                   (__nv_bfloat16*)out, n, act);
    MRUN_CHECK_LAUNCH("plain_act");
    return 0;
}
