// The walk of a recurrence whose read-out does not feed back into its state (a bonus or a state-space
// scan, see recurrent.cu for the formulas), for key sizes that are a multiple of 8 and value sizes
// that are a multiple of 4.
//
// Four warps walk, four bring their input and four collect their output.  A walking lane holds a tile of 8 key rows x CL value columns of
// the head's state in registers, as pairs of rows, so that every step is packed 32-bit arithmetic (two
// multiply-adds an instruction) and the rows of k, q (and g) that a lane reads from shared memory
// serve CL columns.  A warp's lanes are R row slices x C = 32 / R column groups; slice r owns rows
// 4r .. 4r+3 and 4R + 4r .. 4R + 4r+3, so the slices' 16-byte reads lie side by side.  What a lane
// adds to a token's read-out goes to shared memory as it is.
//
// The bringing warps ask global memory for the rows two stages of tokens ahead (two sets of registers in
// turn) and turn those of the next stage into 32-bit rows in shared memory (decays, steps and products
// with the step formed there); the collecting warps add the slices' shares of the stage before, in
// slice order.  The three meet at one barrier a stage.
// There is no kernel in front and no scratch memory.  Nothing in a token's arithmetic depends on the
// tile, on the stage or on how a request was cut into steps.
// grid: value-column groups x heads x segments; a segment of zero rows is padding.  A step of single
// tokens has a smaller kernel of its own, below.
#include "recurrent_walk.h"

#include "common.cuh"

using namespace mrun;

namespace {

constexpr int WARPS = 4;            // of each of the three roles
constexpr int ROLE = WARPS * 32, THREADS = 3 * ROLE;
constexpr int STAGE = 16;           // tokens a stage holds at most
constexpr int CHUNKS = 2;           // chunks of 8 key features a bringing thread carries a vector and stage

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
// Where the roles meet: every thread of the block, from each side of the branch.
__device__ __forceinline__ void stage_barrier() { asm volatile("bar.sync 1, %0;" ::"n"(THREADS) : "memory"); }
__device__ __forceinline__ float2 both(float v) { return make_float2(v, v); }

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

template <typename TA> struct Raw4;
template <> struct Raw4<float> {
    float4 a;
    __device__ __forceinline__ void load(const float* p) { a = load4(p); }
    __device__ __forceinline__ float4 widen() const { return a; }
};
template <> struct Raw4<__nv_bfloat16> {
    uint2 a;
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { a = *reinterpret_cast<const uint2*>(p); }
    __device__ __forceinline__ float4 widen() const {
        const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.x));
        const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.y));
        return make_float4(lo.x, lo.y, hi.x, hi.y);
    }
};

// ------------------------------------------------------------------------------------------
// What both kernels do with a lane's tile: rows of pair p, and columns col .. col + CL - 1.
// ------------------------------------------------------------------------------------------
template <int R> __device__ __forceinline__ int pair_row(int r, int p) { return (p >> 1) * 4 * R + 4 * r + (p & 1) * 2; }

template <int CL> __device__ __forceinline__ void load_columns(const float* p, float (&x)[CL]) {
    if constexpr (CL == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        x[0] = t.x; x[1] = t.y; x[2] = t.z; x[3] = t.w;
    } else if constexpr (CL == 2) {
        const float2 t = *reinterpret_cast<const float2*>(p);
        x[0] = t.x; x[1] = t.y;
    } else {
        x[0] = p[0];
    }
}
template <int CL> __device__ __forceinline__ void store_columns(float* p, const float (&x)[CL]) {
    if constexpr (CL == 4) *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
    else if constexpr (CL == 2) *reinterpret_cast<float2*>(p) = make_float2(x[0], x[1]);
    else p[0] = x[0];
}

template <int R, int CL>
__device__ __forceinline__ void load_tile(const float* st, int r, bool live, int D, int V, float2 (&S)[4][CL]) {
#pragma unroll
    for (int p = 0; p < 4; ++p) {
        const int row = pair_row<R>(r, p);
#pragma unroll
        for (int j = 0; j < CL; ++j) S[p][j] = make_float2(0.f, 0.f);
        if (live && row < D) {
            float x[CL], y[CL];
            load_columns<CL>(st + (size_t)row * V, x);
            load_columns<CL>(st + (size_t)(row + 1) * V, y);
#pragma unroll
            for (int j = 0; j < CL; ++j) S[p][j] = make_float2(x[j], y[j]);
        }
    }
}
template <int R, int CL>
__device__ __forceinline__ void store_tile(float* st, int r, bool live, int D, int V, const float2 (&S)[4][CL]) {
#pragma unroll
    for (int p = 0; p < 4; ++p) {
        const int row = pair_row<R>(r, p);
        if (live && row < D) {
            float x[CL], y[CL];
#pragma unroll
            for (int j = 0; j < CL; ++j) { x[j] = S[p][j].x; y[j] = S[p][j].y; }
            store_columns<CL>(st + (size_t)row * V, x);
            store_columns<CL>(st + (size_t)(row + 1) * V, y);
        }
    }
}

// One token: the state advances, o gets the tile's share of the read-out.  gg: the decays of the pairs
// (bonus), or the head's in gg[0] (state space).
template <int MODE, int CL>
__device__ __forceinline__ void advance(float2 (&S)[4][CL], const float2 (&qq)[4], const float2 (&kk)[4],
                                        const float2 (&gg)[4], const float2 (&u)[4], const float (&vv)[CL], float (&o)[CL]) {
    // neighbouring columns' steps stand side by side: none waits for the one before
    float2 v2[CL], acc[CL];
#pragma unroll
    for (int j = 0; j < CL; ++j) {
        v2[j] = both(vv[j]);
        acc[j] = make_float2(0.f, 0.f);
    }
#pragma unroll
    for (int p = 0; p < 4; ++p) {
        float2 write[CL];
#pragma unroll
        for (int j = 0; j < CL; ++j) write[j] = __fmul2_rn(kk[p], v2[j]);
        if constexpr (MODE == WALK_BONUS) {             // the state before this token's write, the write weighed by u
            float2 seen[CL];
#pragma unroll
            for (int j = 0; j < CL; ++j) seen[j] = __ffma2_rn(u[p], write[j], S[p][j]);
#pragma unroll
            for (int j = 0; j < CL; ++j) S[p][j] = __ffma2_rn(gg[p], S[p][j], write[j]);
#pragma unroll
            for (int j = 0; j < CL; ++j) acc[j] = __ffma2_rn(seen[j], qq[p], acc[j]);
        } else {
#pragma unroll
            for (int j = 0; j < CL; ++j) S[p][j] = __ffma2_rn(gg[0], S[p][j], write[j]);
#pragma unroll
            for (int j = 0; j < CL; ++j) acc[j] = __ffma2_rn(S[p][j], qq[p], acc[j]);
        }
    }
#pragma unroll
    for (int j = 0; j < CL; ++j) o[j] = acc[j].x + acc[j].y;
}

// Floats of the shared-memory areas: a stage's input rows, and the slices' shares of its read-outs (a
// walking warp's start C * CL banks after the one's before, so that a row of columns is read without conflicts).
template <int MODE, int R, int CL> __host__ __device__ constexpr int input_floats(int stage) {
    return stage * ((MODE == WALK_BONUS ? 3 : 2) * 8 * R + WARPS * (32 / R) * CL) + STAGE;
}
template <int R, int CL> constexpr int SHARE_WARP = 32 * CL + (32 / R) * CL;

template <typename TA, int MODE, int R, int CL>
__global__ void __launch_bounds__(THREADS, 1)
walk_kernel(const WalkArgs w) {
    constexpr bool BONUS = MODE == WALK_BONUS;
    constexpr int C = 32 / R, COLS = WARPS * C * CL, ROWS = 8 * R;
    constexpr int VECTORS = BONUS ? 3 : 2;
    constexpr int V_CHUNKS = (STAGE * COLS / 4 + ROLE - 1) / ROLE;
    extern __shared__ __align__(16) float smem[];       // [2] input rows, [2] shares
    const int tid = threadIdx.x;
    const int h = blockIdx.y, seg = blockIdx.z;
    const int q0 = w.seg_q_start[seg], n = w.seg_q_start[seg + 1] - q0;
    if (n <= 0) return;
    const int D = w.D, V = w.V, H = w.H, stage = w.stage;
    const int block_col = blockIdx.x * COLS;
    const int buffer = input_floats<MODE, R, CL>(stage), shares = stage * WARPS * SHARE_WARP<R, CL>;
    const int stages = (n + stage - 1) / stage;

    if (D < ROWS) {                                     // rows beyond the key size stay zero: their state does too
        for (int i = tid; i < 2 * buffer; i += THREADS) smem[i] = 0.f;
        __syncthreads();
    }
    if (tid < ROLE) {
        // ------------------------------------------------------------------------------ the walk
        const int lane = tid & 31, warp = tid >> 5;
        const int r = lane / C, c = lane % C;
        const int my_col = (warp * C + c) * CL, col = block_col + my_col;
        const bool live = col < V;                      // V is a multiple of CL
        float2 S[4][CL], u[4];
        float* st = w.state + (((size_t)w.seg_slot[seg] * H + h) * D) * V + col;
        load_tile<R, CL>(st, r, live, D, V, S);
#pragma unroll
        for (int p = 0; p < 4; ++p) {
            const int row = pair_row<R>(r, p);
            u[p] = make_float2(0.f, 0.f);
            if (BONUS && row < D) u[p] = *reinterpret_cast<const float2*>(w.bonus + (size_t)h * D + row);
        }
        stage_barrier();                                // the first stage's rows are there
        for (int s = 0; s < stages; ++s) {
            const int m = min(stage, n - s * stage);
            const float* base = smem + (s & 1) * buffer;
            float* share = smem + 2 * buffer + (s & 1) * shares + warp * SHARE_WARP<R, CL> + lane * CL;
#pragma unroll 4
            for (int t = 0; t < m; ++t) {
                const float4* q4 = reinterpret_cast<const float4*>(base + t * ROWS);
                const float4* k4 = reinterpret_cast<const float4*>(base + (stage + t) * ROWS);
                [[maybe_unused]] const float4* g4 = reinterpret_cast<const float4*>(base + (2 * stage + t) * ROWS);
                float vv[CL];
                const float* vs = base + VECTORS * stage * ROWS + t * COLS + my_col;
                load_columns<CL>(vs, vv);
                const float4 qa = q4[r], qb = q4[R + r], ka = k4[r], kb = k4[R + r];
                const float2 qq[4] = {{qa.x, qa.y}, {qa.z, qa.w}, {qb.x, qb.y}, {qb.z, qb.w}};
                const float2 kk[4] = {{ka.x, ka.y}, {ka.z, ka.w}, {kb.x, kb.y}, {kb.z, kb.w}};
                float2 gg[4];
                if constexpr (BONUS) {
                    const float4 ga = g4[r], gb = g4[R + r];
                    gg[0] = {ga.x, ga.y}; gg[1] = {ga.z, ga.w}; gg[2] = {gb.x, gb.y}; gg[3] = {gb.z, gb.w};
                } else {
                    gg[0] = both(base[VECTORS * stage * ROWS + stage * COLS + t]);
                }
                float o[CL];
                advance<MODE, CL>(S, qq, kk, gg, u, vv, o);
                store_columns<CL>(share + t * (WARPS * SHARE_WARP<R, CL>), o);
            }
            stage_barrier();
        }
        store_tile<R, CL>(st, r, live, D, V, S);
    } else if (tid < 2 * ROLE) {
        // ------------------------------------------------------------------------- bringing input
        const int me = tid - ROLE;
        const int kh = h / w.group;
        const TA* q = (const TA*)w.q + (size_t)q0 * w.ld + (size_t)kh * D;
        const TA* k = (const TA*)w.k + (size_t)q0 * w.ld + (size_t)kh * D;
        const TA* v = (const TA*)w.v + (size_t)q0 * w.ld + (size_t)h * V + block_col;
        const float* a = BONUS ? w.a + ((size_t)q0 * H + h) * D : nullptr;
        const TA* dt = BONUS ? nullptr : (const TA*)w.dt + (size_t)q0 * w.lddt + h;
        const float dt_bias = BONUS ? 0.f : w.bias[h], rate = BONUS ? 0.f : expf(w.a_log[h]);
        const int row_chunks = D >> 3;
        struct Rows {                                   // of one stage, as they lie in memory
            Raw8<TA> q[CHUNKS], k[CHUNKS];
            Raw8<float> a[BONUS ? CHUNKS : 1];
            Raw4<TA> v[V_CHUNKS];
            TA dt[V_CHUNKS], dt_head;
        } even, odd;
        auto fetch = [&](int s, Rows& x) {              // stage s: from global memory to registers
            if (s >= stages) return;
            const int t0 = s * stage, m = min(stage, n - t0), total = m * row_chunks;
#pragma unroll
            for (int i = 0; i < CHUNKS; ++i) {
                const int e = me + i * ROLE;
                if (e < total) {
                    const int t = e / row_chunks, at = (e - t * row_chunks) * 8;
                    const size_t off = (size_t)(t0 + t) * w.ld + at;
                    x.q[i].load(q + off);
                    x.k[i].load(k + off);
                    if constexpr (BONUS) x.a[i].load(a + (size_t)(t0 + t) * H * D + at);
                }
            }
#pragma unroll
            for (int i = 0; i < V_CHUNKS; ++i) {
                const int e = me + i * ROLE, t = e / (COLS / 4), j = (e % (COLS / 4)) * 4;
                if (t < m && block_col + j < V) {
                    x.v[i].load(v + (size_t)(t0 + t) * w.ld + j);
                    if constexpr (!BONUS) x.dt[i] = dt[(size_t)(t0 + t) * w.lddt];
                }
            }
            if (!BONUS && me < m) x.dt_head = dt[(size_t)(t0 + me) * w.lddt];
        };
        auto settle = [&](int s, const Rows& x) {       // and from there to shared memory, in 32-bit
            if (s >= stages) return;
            const int m = min(stage, n - s * stage), total = m * row_chunks;
            float* qs = smem + (s & 1) * buffer;
            float* ks = qs + stage * ROWS;
            float* gs = ks + stage * ROWS;
            float* vs = qs + VECTORS * stage * ROWS;
            float* ns = vs + stage * COLS;
#pragma unroll
            for (int i = 0; i < CHUNKS; ++i) {
                const int e = me + i * ROLE;
                if (e < total) {
                    const int t = e / row_chunks, at = (e - t * row_chunks) * 8;
                    float y[8];
                    x.q[i].widen(y);
                    Vec8<float>::store(qs + t * ROWS + at, y);
                    x.k[i].widen(y);
                    Vec8<float>::store(ks + t * ROWS + at, y);
                    if constexpr (BONUS) {
                        float b[8];
                        x.a[i].widen(y);
                        Vec8<float>::load(w.bias + (size_t)h * D + at, b);
#pragma unroll
                        for (int j = 0; j < 8; ++j) y[j] = expf(-expf(y[j] + b[j]));
                        Vec8<float>::store(gs + t * ROWS + at, y);
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < V_CHUNKS; ++i) {
                const int e = me + i * ROLE, t = e / (COLS / 4), j = (e % (COLS / 4)) * 4;
                if (t < m && block_col + j < V) {
                    float4 y = x.v[i].widen();
                    if constexpr (!BONUS) {
                        const float step = softplus_f(to_float(x.dt[i]) + dt_bias);
                        y.x *= step; y.y *= step; y.z *= step; y.w *= step;
                    }
                    *reinterpret_cast<float4*>(vs + t * COLS + j) = y;
                }
            }
            if (!BONUS && me < m) ns[me] = expf(-rate * softplus_f(to_float(x.dt_head) + dt_bias));
        };
        fetch(0, even);
        fetch(1, odd);
        settle(0, even);
        fetch(2, even);
        stage_barrier();
        for (int s = 0; s < stages; s += 2) {           // (a buffer was walked before the last barrier)
            settle(s + 1, odd);
            fetch(s + 3, odd);
            stage_barrier();
            if (s + 1 == stages) break;
            settle(s + 2, even);
            fetch(s + 4, even);
            stage_barrier();
        }
    } else {
        // ----------------------------------------------------------------------- collecting output
        const int me = tid - 2 * ROLE;
        float* out = w.out + (size_t)q0 * H * V + (size_t)h * V + block_col;
        auto gather = [&](int s) {                      // the slices' shares of stage s, added in slice order
            const int t0 = s * stage, m = min(stage, n - t0);
            const float* base = smem + 2 * buffer + (s & 1) * shares;
#pragma unroll 2
            for (int e = me; e < m * COLS; e += ROLE) {
                const int t = e / COLS, j = e % COLS;
                if (block_col + j >= V) continue;
                const float* from = base + (t * WARPS + j / (C * CL)) * SHARE_WARP<R, CL> + j % (C * CL);
                float x[R];
#pragma unroll
                for (int i = 0; i < R; ++i) x[i] = from[i * C * CL];
#pragma unroll
                for (int i = 1; i < R; ++i) x[0] += x[i];
                out[(size_t)(t0 + t) * H * V + j] = x[0];
            }
        };
        stage_barrier();
        for (int s = 0; s < stages; ++s) {
            if (s > 0) gather(s - 1);
            stage_barrier();
        }
        gather(stages - 1);
    }
}

// ------------------------------------------------------------------------------------------
// The same for a step in which every segment is a single token (or none): the state's tile is asked for
// first, a lane makes its own rows of q, k and the decays, the slices' shares meet in shared memory
// once.  Nothing is staged and a block is four warps, so that many tiles are in flight; the arithmetic
// and the order of the sums are the walk's.
// ------------------------------------------------------------------------------------------
template <typename TA, int MODE, int R, int CL>
__global__ void __launch_bounds__(ROLE)
single_kernel(const WalkArgs w) {
    constexpr bool BONUS = MODE == WALK_BONUS;
    constexpr int C = 32 / R, COLS = WARPS * C * CL;
    __shared__ __align__(16) float shares[WARPS * SHARE_WARP<R, CL>];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, seg = blockIdx.z;
    const int q0 = w.seg_q_start[seg];
    if (w.seg_q_start[seg + 1] <= q0) return;
    const int D = w.D, V = w.V, H = w.H;
    const int block_col = blockIdx.x * COLS;
    const int r = lane / C, c = lane % C, col = block_col + (warp * C + c) * CL;
    const bool live = col < V;
    float2 S[4][CL];
    float* st = w.state + (((size_t)w.seg_slot[seg] * H + h) * D) * V + col;
    load_tile<R, CL>(st, r, live, D, V, S);
    float2 qq[4], kk[4], gg[4], u[4];
    const int kh = h / w.group;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int row = half * 4 * R + 4 * r;           // pairs 2 half and 2 half + 1
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x, g = x, b = x;
        if (row < D) {
            Raw4<TA> raw;
            raw.load((const TA*)w.q + (size_t)q0 * w.ld + (size_t)kh * D + row);
            x = raw.widen();
            raw.load((const TA*)w.k + (size_t)q0 * w.ld + (size_t)kh * D + row);
            y = raw.widen();
            if constexpr (BONUS) {
                const float4 z = load4(w.a + ((size_t)q0 * H + h) * D + row), bias = load4(w.bias + (size_t)h * D + row);
                g = make_float4(expf(-expf(z.x + bias.x)), expf(-expf(z.y + bias.y)), expf(-expf(z.z + bias.z)), expf(-expf(z.w + bias.w)));
                b = load4(w.bonus + (size_t)h * D + row);
            }
        }
        qq[2 * half] = make_float2(x.x, x.y); qq[2 * half + 1] = make_float2(x.z, x.w);
        kk[2 * half] = make_float2(y.x, y.y); kk[2 * half + 1] = make_float2(y.z, y.w);
        gg[2 * half] = make_float2(g.x, g.y); gg[2 * half + 1] = make_float2(g.z, g.w);
        u[2 * half] = make_float2(b.x, b.y); u[2 * half + 1] = make_float2(b.z, b.w);
    }
    float step = 1.f;
    if constexpr (!BONUS) {
        step = softplus_f(to_float(((const TA*)w.dt)[(size_t)q0 * w.lddt + h]) + w.bias[h]);
        gg[0] = both(expf(-expf(w.a_log[h]) * step));
    }
    float vv[CL], o[CL];
#pragma unroll
    for (int j = 0; j < CL; ++j) vv[j] = live ? to_float(((const TA*)w.v)[(size_t)q0 * w.ld + (size_t)h * V + col + j]) * step : 0.f;
    advance<MODE, CL>(S, qq, kk, gg, u, vv, o);
    store_columns<CL>(shares + warp * SHARE_WARP<R, CL> + lane * CL, o);
    store_tile<R, CL>(st, r, live, D, V, S);
    __syncthreads();
    for (int j = tid; j < COLS; j += ROLE) {
        if (block_col + j >= V) continue;
        const float* from = shares + (j / (C * CL)) * SHARE_WARP<R, CL> + j % (C * CL);
        float x[R];
#pragma unroll
        for (int i = 0; i < R; ++i) x[i] = from[i * C * CL];
#pragma unroll
        for (int i = 1; i < R; ++i) x[0] += x[i];
        w.out[(size_t)q0 * H * V + (size_t)h * V + block_col + j] = x[0];
    }
}

template <typename TA, int MODE, int R, int CL>
int launch(WalkArgs w, int segments, cudaStream_t stream) {
    constexpr int COLS = WARPS * (32 / R) * CL;
    if (w.max_q_len == 1) {
        single_kernel<TA, MODE, R, CL><<<dim3((w.V + COLS - 1) / COLS, w.H, segments), ROLE, 0, stream>>>(w);
        MRUN_CHECK_LAUNCH("scan step");
        return 0;
    }
    const int carried = CHUNKS * ROLE * 8 / w.D;     // tokens whose chunks the bringing threads carry
    w.stage = carried > STAGE ? STAGE : carried / 4 * 4;
    const size_t smem = sizeof(float) * 2 * ((size_t)input_floats<MODE, R, CL>(w.stage) + (size_t)w.stage * WARPS * SHARE_WARP<R, CL>);
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
