// The walk of a recurrence whose read-out does not feed back into its state (a bonus or a state-space
// scan, see recurrent.cu for the formulas), for key sizes that are a multiple of 8 and value sizes
// that are a multiple of 4.
//
// A lane holds a tile of 8 key rows x CL value columns of the head's state in registers, as pairs of
// rows, so that every step is packed 32-bit arithmetic (two multiply-adds an instruction) and the rows
// of k, q (and g) that a lane reads from shared memory serve CL columns.  A warp's lanes are R row
// slices x C = 32 / R column groups; slice r owns rows 4r .. 4r+3 and 4R + 4r .. 4R + 4r+3, so the
// slices' 16-byte reads lie side by side.  Tokens are walked four at a time: their partial read-outs
// meet across the slices together, half of the values handed over at every step instead of all of
// them kept by both sides.  Additions pair the same slices in the same order whatever the tile, the
// number of tokens walked together or the step's cut, so a token's result has the same bits in all.
//
// The rows of the next tokens travel from global memory to registers under the walk over the present
// ones and are turned into 32-bit rows in shared memory (decays, steps and products with the step
// formed there) behind it; there is no kernel in front and no scratch memory.
// grid: value-column groups x heads x segments; a segment of zero rows is padding.
#include "recurrent_walk.h"

#include "common.cuh"

using namespace mrun;

namespace {

constexpr int WARPS = 4, THREADS = WARPS * 32;
constexpr int STAGE = 16;           // tokens a stage holds at most
constexpr int CHUNKS = 2;           // chunks of 8 key features a thread carries a vector and stage

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float2 both(float v) { return make_float2(v, v); }

// NV values a lane, summed over the slices (lane bits from `STEP` lanes upwards, R of them): while a lane
// has more than one value the two sides of a step share them out; v[0 .. max(1, NV / R)) is the lane's
// share afterwards.
template <int NV, int OFF, int STEP>
__device__ __forceinline__ void reduce_slices(float* v, int lane) {
    if constexpr (OFF >= STEP) {
        if constexpr (NV > 1) {
            const bool up = lane & OFF;
#pragma unroll
            for (int i = 0; i < NV / 2; ++i) {
                const float give = up ? v[i] : v[i + NV / 2], keep = up ? v[i + NV / 2] : v[i];
                v[i] = keep + __shfl_xor_sync(0xffffffffu, give, OFF);
            }
            reduce_slices<NV / 2, OFF / 2, STEP>(v, lane);
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], OFF);
            reduce_slices<1, OFF / 2, STEP>(v, lane);
        }
    }
}

template <typename TA> struct Raw8;                 // eight features as they lie in memory
template <> struct Raw8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) {
        a = *reinterpret_cast<const float4*>(p);
        b = *reinterpret_cast<const float4*>(p + 4);
    }
    __device__ __forceinline__ void widen(float (&v)[8]) const {
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    }
};
template <> struct Raw8<__nv_bfloat16> {
    uint4 a;
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { a = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ void widen(float (&v)[8]) const {
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&a);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(h[i]);
            v[2 * i] = f.x; v[2 * i + 1] = f.y;
        }
    }
};
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}

template <typename TA, int MODE, int R, int CL>
__global__ void __launch_bounds__(THREADS)
walk_kernel(const WalkArgs w) {
    constexpr bool BONUS = MODE == WALK_BONUS;
    constexpr int C = 32 / R, COLS = WARPS * C * CL, ROWS = 8 * R;
    constexpr int VECTORS = BONUS ? 3 : 2;
    constexpr int V_CHUNKS = (STAGE * COLS / 4 + THREADS - 1) / THREADS;
    extern __shared__ __align__(16) float smem[];       // [2][VECTORS * stage * ROWS | stage * COLS | stage]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, seg = blockIdx.z;
    const int q0 = w.seg_q_start[seg], n = w.seg_q_start[seg + 1] - q0;
    if (n <= 0) return;
    const int D = w.D, V = w.V, H = w.H, stage = w.stage;
    const int r = lane / C, c = lane % C;
    const int block_col = blockIdx.x * COLS, my_col = (warp * C + c) * CL, col = block_col + my_col;
    const bool live = col < V;                          // V is a multiple of CL
    const int kh = h / w.group;
    const int buffer = stage * (VECTORS * ROWS + COLS) + STAGE;
    const TA* q = (const TA*)w.q + (size_t)q0 * w.ld + (size_t)kh * D;
    const TA* k = (const TA*)w.k + (size_t)q0 * w.ld + (size_t)kh * D;
    const TA* v = (const TA*)w.v + (size_t)q0 * w.ld + (size_t)h * V + block_col;
    const float* a = BONUS ? w.a + ((size_t)q0 * H + h) * D : nullptr;
    const TA* dt = BONUS ? nullptr : (const TA*)w.dt + (size_t)q0 * w.lddt + h;
    const float dt_bias = BONUS ? 0.f : w.bias[h], rate = BONUS ? 0.f : expf(w.a_log[h]);

    if (D < ROWS)                                       // rows beyond the key size stay zero: their state does too
        for (int i = tid; i < 2 * buffer; i += THREADS) smem[i] = 0.f;

    // ---------------------------------------------------------------- state
    auto row_of = [&](int p) { return (p >> 1) * 4 * R + 4 * r + (p & 1) * 2; };      // first row of pair p
    float2 S[4][CL], u[4];
    float* st = w.state + (((size_t)w.seg_slot[seg] * H + h) * D) * V + col;
#pragma unroll
    for (int p = 0; p < 4; ++p) {
        const int row = row_of(p);
        const bool mine = live && row < D;
#pragma unroll
        for (int j = 0; j < CL; ++j) S[p][j] = make_float2(0.f, 0.f);
        if (mine) {
            float x[CL], y[CL];
            if constexpr (CL == 4) {
                *reinterpret_cast<float4*>(x) = load4(st + (size_t)row * V);
                *reinterpret_cast<float4*>(y) = load4(st + (size_t)(row + 1) * V);
            } else if constexpr (CL == 2) {
                *reinterpret_cast<float2*>(x) = *reinterpret_cast<const float2*>(st + (size_t)row * V);
                *reinterpret_cast<float2*>(y) = *reinterpret_cast<const float2*>(st + (size_t)(row + 1) * V);
            } else {
                x[0] = st[(size_t)row * V];
                y[0] = st[(size_t)(row + 1) * V];
            }
#pragma unroll
            for (int j = 0; j < CL; ++j) S[p][j] = make_float2(x[j], y[j]);
        }
        u[p] = make_float2(0.f, 0.f);
        if (BONUS && row < D) u[p] = *reinterpret_cast<const float2*>(w.bonus + (size_t)h * D + row);
    }

    // ---------------------------------------------------------------- rows of the coming tokens
    Raw8<TA> rq[CHUNKS], rk[CHUNKS];
    Raw8<float> ra[BONUS ? CHUNKS : 1];
    float4 rv[V_CHUNKS];
    float rdt[V_CHUNKS], rdt_head = 0.f;
    const int row_chunks = D >> 3;
    auto fetch = [&](int t0) {
        const int m = min(stage, n - t0), total = m * row_chunks;
#pragma unroll
        for (int i = 0; i < CHUNKS; ++i) {
            const int e = tid + i * THREADS;
            if (e < total) {
                const int t = e / row_chunks, at = (e - t * row_chunks) * 8;
                const size_t off = (size_t)(t0 + t) * w.ld + at;
                rq[i].load(q + off);
                rk[i].load(k + off);
                if constexpr (BONUS) ra[i].load(a + (size_t)(t0 + t) * H * D + at);
            }
        }
#pragma unroll
        for (int i = 0; i < V_CHUNKS; ++i) {
            const int e = tid + i * THREADS, t = e / (COLS / 4), j = (e % (COLS / 4)) * 4;
            if (t < m && block_col + j < V) {
                rv[i] = load4(v + (size_t)(t0 + t) * w.ld + j);
                if constexpr (!BONUS) rdt[i] = to_float(dt[(size_t)(t0 + t) * w.lddt]);
            }
        }
        if (!BONUS && tid < m) rdt_head = to_float(dt[(size_t)(t0 + tid) * w.lddt]);
    };
    auto settle = [&](int which, int t0) {
        const int m = min(stage, n - t0), total = m * row_chunks;
        float* qs = smem + which * buffer;
        float* ks = qs + stage * ROWS;
        float* gs = ks + stage * ROWS;
        float* vs = qs + VECTORS * stage * ROWS;
        float* ns = vs + stage * COLS;
#pragma unroll
        for (int i = 0; i < CHUNKS; ++i) {
            const int e = tid + i * THREADS;
            if (e < total) {
                const int t = e / row_chunks, at = (e - t * row_chunks) * 8;
                float x[8];
                rq[i].widen(x);
                Vec8<float>::store(qs + t * ROWS + at, x);
                rk[i].widen(x);
                Vec8<float>::store(ks + t * ROWS + at, x);
                if constexpr (BONUS) {
                    float b[8];
                    ra[i].widen(x);
                    Vec8<float>::load(w.bias + (size_t)h * D + at, b);
#pragma unroll
                    for (int j = 0; j < 8; ++j) x[j] = expf(-expf(x[j] + b[j]));
                    Vec8<float>::store(gs + t * ROWS + at, x);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < V_CHUNKS; ++i) {
            const int e = tid + i * THREADS, t = e / (COLS / 4), j = (e % (COLS / 4)) * 4;
            if (t < m && block_col + j < V) {
                float4 x = rv[i];
                if constexpr (!BONUS) {
                    const float step = softplus_f(rdt[i] + dt_bias);
                    x.x *= step; x.y *= step; x.z *= step; x.w *= step;
                }
                *reinterpret_cast<float4*>(vs + t * COLS + j) = x;
            }
        }
        if (!BONUS && tid < m) ns[tid] = expf(-rate * softplus_f(rdt_head + dt_bias));
    };

    // ---------------------------------------------------------------- NT tokens from row tt of a stage
    auto walk = [&](auto count, int which, int tt, int t0) {
        constexpr int NT = decltype(count)::value;
        const float* base = smem + which * buffer;
        float o[NT * CL];
#pragma unroll
        for (int t = 0; t < NT; ++t) {
            const float4* q4 = reinterpret_cast<const float4*>(base + (tt + t) * ROWS);
            const float4* k4 = reinterpret_cast<const float4*>(base + (stage + tt + t) * ROWS);
            [[maybe_unused]] const float4* g4 = reinterpret_cast<const float4*>(base + (2 * stage + tt + t) * ROWS);
            float vv[CL];
            const float* vs = base + VECTORS * stage * ROWS + (tt + t) * COLS + my_col;
            if constexpr (CL == 4) *reinterpret_cast<float4*>(vv) = *reinterpret_cast<const float4*>(vs);
            else if constexpr (CL == 2) *reinterpret_cast<float2*>(vv) = *reinterpret_cast<const float2*>(vs);
            else vv[0] = vs[0];
            const float4 qa = q4[r], qb = q4[R + r], ka = k4[r], kb = k4[R + r];
            const float2 qq[4] = {{qa.x, qa.y}, {qa.z, qa.w}, {qb.x, qb.y}, {qb.z, qb.w}};
            const float2 kk[4] = {{ka.x, ka.y}, {ka.z, ka.w}, {kb.x, kb.y}, {kb.z, kb.w}};
            float2 gg[4];
            if constexpr (BONUS) {
                const float4 ga = g4[r], gb = g4[R + r];
                gg[0] = {ga.x, ga.y}; gg[1] = {ga.z, ga.w}; gg[2] = {gb.x, gb.y}; gg[3] = {gb.z, gb.w};
            } else {
                gg[0] = both(base[VECTORS * stage * ROWS + stage * COLS + tt + t]);
            }
#pragma unroll
            for (int j = 0; j < CL; ++j) {
                const float2 v2 = both(vv[j]);
                float2 acc = make_float2(0.f, 0.f);
#pragma unroll
                for (int p = 0; p < 4; ++p) {
                    const float2 write = __fmul2_rn(kk[p], v2);
                    if constexpr (BONUS) {              // the state before this token's write, the write weighed by u
                        acc = __ffma2_rn(__ffma2_rn(u[p], write, S[p][j]), qq[p], acc);
                        S[p][j] = __ffma2_rn(gg[p], S[p][j], write);
                    } else {
                        S[p][j] = __ffma2_rn(gg[0], S[p][j], write);
                        acc = __ffma2_rn(S[p][j], qq[p], acc);
                    }
                }
                o[t * CL + j] = acc.x + acc.y;
            }
        }
        reduce_slices<NT * CL, 16, C>(o, lane);
        // the lane's share: NV / R values from number r * (NV / R) on, or (NV < R) value r / (R / NV)
        constexpr int NV = NT * CL, SHARE = NV > R ? NV / R : 1, OWNERS = NV < R ? R / NV : 1;
        if (live && r % OWNERS == 0) {
#pragma unroll
            for (int i = 0; i < SHARE; ++i) {
                const int number = (r / OWNERS) * SHARE + i;
                w.out[(size_t)(q0 + t0 + tt + number / CL) * H * V + (size_t)h * V + col + number % CL] = o[i];
            }
        }
    };

    fetch(0);
    __syncthreads();                                    // the zero fill comes before the rows
    settle(0, 0);
    __syncthreads();
    int which = 0;
    for (int t0 = 0; t0 < n; t0 += stage, which ^= 1) {
        const int m = min(stage, n - t0);
        const bool more = t0 + stage < n;
        if (more) fetch(t0 + stage);
        int tt = 0;
        for (; tt + 4 <= m; tt += 4) walk(Count<4>{}, which, tt, t0);
        for (; tt < m; ++tt) walk(Count<1>{}, which, tt, t0);
        if (more) settle(which ^ 1, t0 + stage);        // that buffer was walked before the last barrier
        __syncthreads();
    }

#pragma unroll
    for (int p = 0; p < 4; ++p) {
        const int row = row_of(p);
        if (live && row < D) {
            float x[CL], y[CL];
#pragma unroll
            for (int j = 0; j < CL; ++j) { x[j] = S[p][j].x; y[j] = S[p][j].y; }
            if constexpr (CL == 4) {
                *reinterpret_cast<float4*>(st + (size_t)row * V) = *reinterpret_cast<float4*>(x);
                *reinterpret_cast<float4*>(st + (size_t)(row + 1) * V) = *reinterpret_cast<float4*>(y);
            } else if constexpr (CL == 2) {
                *reinterpret_cast<float2*>(st + (size_t)row * V) = *reinterpret_cast<float2*>(x);
                *reinterpret_cast<float2*>(st + (size_t)(row + 1) * V) = *reinterpret_cast<float2*>(y);
            } else {
                st[(size_t)row * V] = x[0];
                st[(size_t)(row + 1) * V] = y[0];
            }
        }
    }
}

template <typename TA, int MODE, int R, int CL>
int launch(WalkArgs w, int segments, cudaStream_t stream) {
    constexpr int COLS = WARPS * (32 / R) * CL, ROWS = 8 * R;
    int stage = CHUNKS * THREADS * 8 / w.D;             // the chunks a thread carries
    w.stage = stage > STAGE ? STAGE : stage / 4 * 4;
    const size_t smem = sizeof(float) * 2 * ((size_t)w.stage * ((MODE == WALK_BONUS ? 3 : 2) * ROWS + COLS) + STAGE);
    if (smem > 48 * 1024)
        MRUN_CHECK_CUDA(cudaFuncSetAttribute(walk_kernel<TA, MODE, R, CL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem),
                        "scan walk");
    walk_kernel<TA, MODE, R, CL><<<dim3((w.V + COLS - 1) / COLS, w.H, segments), THREADS, smem, stream>>>(w);
    MRUN_CHECK_LAUNCH("scan walk");
    return 0;
}

// Columns a lane holds: the widest tile that still leaves a block for most multiprocessors (a function of
// the launch's shape; the results do not depend on it).
template <typename TA, int MODE>
int dispatch(const WalkArgs& w, int segments, cudaStream_t stream) {
    const int slices = (w.D + 7) / 8;
    auto blocks = [&](int R, int CL) { return (long)((w.V + WARPS * (32 / R) * CL - 1) / (WARPS * (32 / R) * CL)) * w.H * segments; };
    constexpr long FULL = 96;
    if (slices <= 1) return launch<TA, MODE, 1, 1>(w, segments, stream);
    if (slices <= 2) return launch<TA, MODE, 2, 1>(w, segments, stream);
    if (slices <= 4) return launch<TA, MODE, 4, 1>(w, segments, stream);
    if (slices <= 8) {
        if (blocks(8, 2) >= FULL) return launch<TA, MODE, 8, 2>(w, segments, stream);
        return launch<TA, MODE, 8, 1>(w, segments, stream);
    }
    if (slices <= 16) {
        if (blocks(16, 4) >= FULL) return launch<TA, MODE, 16, 4>(w, segments, stream);
        return launch<TA, MODE, 16, 2>(w, segments, stream);
    }
    if (blocks(32, 4) >= FULL) return launch<TA, MODE, 32, 4>(w, segments, stream);
    return launch<TA, MODE, 32, 2>(w, segments, stream);
}

}  // namespace

bool walk_takes(const WalkArgs& w, int act_dtype) {
    const size_t unit = act_dtype == MRUN_F32 ? 4 : 2;
    return (act_dtype == MRUN_F32 || act_dtype == MRUN_BF16) && w.D % 8 == 0 && w.D <= 256 && w.V % 4 == 0 &&
           (w.ld * unit) % 16 == 0 && (((uintptr_t)w.q | (uintptr_t)w.k) & 15) == 0 && ((uintptr_t)w.v & (4 * unit - 1)) == 0 &&
           (((uintptr_t)w.a | (uintptr_t)w.bonus | (uintptr_t)w.state) & 15) == 0 &&
           (w.mode != WALK_BONUS || ((uintptr_t)w.bias & 15) == 0);
}

int launch_walk(const WalkArgs& w, int act_dtype, int segments, cudaStream_t stream) {
    if (act_dtype == MRUN_F32)
        return w.mode == WALK_BONUS ? dispatch<float, WALK_BONUS>(w, segments, stream) : dispatch<float, WALK_SSM>(w, segments, stream);
    return w.mode == WALK_BONUS ? dispatch<__nv_bfloat16, WALK_BONUS>(w, segments, stream)
                                : dispatch<__nv_bfloat16, WALK_SSM>(w, segments, stream);
}
