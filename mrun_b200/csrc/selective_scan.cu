// The selective scan of a state-space mixer whose decays belong to channels and states (Mamba): per
// request, channel c and state n, over the request's tokens,
//
//   step_c = softplus(dt_c + bias_c)
//   S[c, n] <- exp(step_c A[c, n]) S[c, n] + step_c x_c B_n
//   out_c   = (sum_n S[c, n] C_n + skip_c x_c) * SiLU(z_c)
//
// from and into the request's state (float32 [inner, states]).  Everything but the rows themselves is 32-bit.
//
// A lane holds NS states of one channel as pairs (packed 32-bit arithmetic), L lanes hold a channel.  Eight
// warps of a block walk; eight others bring the input of the stage ahead and carry the finished rows of the
// stage behind to memory.  Rows of x, z and dt are asked for two stages ahead and become (step, step * x) in
// shared memory and (skip * x, SiLU(z)) in the registers of the thread that later finishes the element; B and
// C, 32-bit rows, are copied two stages ahead into a ring of three, the pairs of a lane side by side.  The
// roles meet at one barrier a stage.  What bounds the walk is shared memory's bandwidth, then the exponentials.
//
// A walking lane's work is the exponential, one a state and token; so four tokens go side by side and their
// read-outs are summed over the channel's lanes together: two exchanges halve the tokens a lane is in
// charge of, so that lane l of the first four ends with token l's sum (three shuffles for four tokens).
// The sum of a token is ((l0 + l1) + (l2 + l3)) + ... whatever its place, a step without a token has step 0
// and leaves the state as it is (decay 1, nothing written), so a token's result has the same bits however its request was
// cut.  A step of single tokens has a smaller kernel with the same arithmetic, which takes B and C in the
// activation type.
// grid: channel groups x segments; a segment of zero rows is padding.
#include "common.cuh"

using namespace mrun;

namespace {

constexpr int WARPS = 8;                    // of each of the two roles
constexpr int ROLE = WARPS * 32, THREADS = 2 * ROLE;
constexpr int SINGLE = 128;                 // threads of a block of the kernel for single tokens

struct ScanArgs {
    const void *x, *z;                      // rows of the activation type
    const void *b, *c;                      // of 32-bit floats; of the activation type in a step of single tokens
    long ldx, ldz, ldbc;
    const float* dt;                        // [tokens, inner], rows lddt apart
    long lddt;
    const float *dt_bias, *a, *skip;        // [inner], [inner, states] (negative), [inner]
    float* state;                           // [slots, inner, states]
    void* out;                              // [tokens, inner], rows ldo apart
    long ldo;
    const int *seg_q_start, *seg_slot;
    int inner, states;
};

__device__ __forceinline__ float exp2_fast(float v) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
    return r;
}
__device__ __forceinline__ float log2_fast(float v) {
    float r;
    asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
    return r;
}
__device__ __forceinline__ float reciprocal_fast(float v) {
    float r;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
    return r;
}
constexpr float LOG2_E = 1.4426950408889634f, LN_2 = 0.6931471805599453f;
// log(1 + e) for e >= 0.  Up to one half by 2 artanh(e / (2 + e)), the odd series through the eleventh power
// (its argument is at most 1/5: the first term left out is below 4e-10 of the sum), so that a small e keeps
// its digits; above by the base-2 logarithm, whose value is not small there.
__device__ __forceinline__ float log1p_fast(float e) {
    const float s = e * reciprocal_fast(2.f + e), z = s * s;
    float p = 2.f / 11.f;
    p = fmaf(p, z, 2.f / 9.f);
    p = fmaf(p, z, 2.f / 7.f);
    p = fmaf(p, z, 2.f / 5.f);
    p = fmaf(p, z, 2.f / 3.f);
    p = fmaf(p, z, 2.f);
    return e <= 0.5f ? s * p : log2_fast(1.f + e) * LN_2;
}
// The 32-bit path calls the library's functions, the 16-bit path works in 32-bit on the fast exponential.
template <typename TA> __device__ __forceinline__ float softplus_f(float x) {
    if constexpr (sizeof(TA) == 4) return x > 20.f ? x : log1pf(expf(x));
    else return x > 20.f ? x : log1p_fast(exp2_fast(x * LOG2_E));
}
template <typename TA> __device__ __forceinline__ float silu_f(float z) {
    if constexpr (sizeof(TA) == 4) return z / (1.f + expf(-z));
    else return z * reciprocal_fast(1.f + exp2_fast(z * -LOG2_E));
}
__device__ __forceinline__ void stage_barrier() { asm volatile("bar.sync 1, %0;" ::"n"(THREADS) : "memory"); }
__device__ __forceinline__ float2 both(float v) { return make_float2(v, v); }
// What a decay's rate is multiplied by when it is loaded: the 16-bit path takes powers of two.
template <typename TA> constexpr float RATE_UNIT = sizeof(TA) == 4 ? 1.f : LOG2_E;

// W consecutive values as they lie in memory (W = 4: one 8- or 16-byte piece).
template <typename TA, int W> struct Piece {
    alignas(sizeof(TA) * W) TA v[W];
    __device__ __forceinline__ void load(const TA* p) {
        if constexpr (W == 4 && sizeof(TA) == 4) *reinterpret_cast<uint4*>(v) = *reinterpret_cast<const uint4*>(p);
        else if constexpr (W == 4) *reinterpret_cast<uint2*>(v) = *reinterpret_cast<const uint2*>(p);
        else v[0] = p[0];
    }
    __device__ __forceinline__ void store(TA* p) const {
        if constexpr (W == 4 && sizeof(TA) == 4) *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(v);
        else if constexpr (W == 4) *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(v);
        else p[0] = v[0];
    }
};

// What a token's step does to the lane's states: the factors, or (32-bit path) what they lack to one, so that
// a decay next to one keeps its digits.
template <typename TA, int NS>
__device__ __forceinline__ void decays(float2 (&d)[NS / 2], const float2 (&rate)[NS / 2], float step) {
#pragma unroll
    for (int i = 0; i < NS / 2; ++i) {
        const float2 arg = __fmul2_rn(both(step), rate[i]);
        if constexpr (sizeof(TA) == 4) d[i] = make_float2(expm1f(arg.x), expm1f(arg.y));
        else d[i] = make_float2(exp2_fast(arg.x), exp2_fast(arg.y));
    }
}
// One token of a lane's states: they advance, the lane's share of the read-out comes back.
template <typename TA, int NS>
__device__ __forceinline__ float advance(float2 (&S)[NS / 2], const float2 (&d)[NS / 2], float input, const float2 (&b)[NS / 2],
                                         const float2 (&c)[NS / 2]) {
    float2 acc = both(0.f);
#pragma unroll
    for (int i = 0; i < NS / 2; ++i) {
        const float2 write = __fmul2_rn(both(input), b[i]);
        if constexpr (sizeof(TA) == 4) S[i] = __fadd2_rn(S[i], __ffma2_rn(d[i], S[i], write));
        else S[i] = __ffma2_rn(d[i], S[i], write);
        acc = __ffma2_rn(S[i], c[i], acc);
    }
    return acc.x + acc.y;
}

template <typename TA, int NS>
__device__ __forceinline__ void load_lane(const ScanArgs& a, const float* st, int ch, int n0, bool live, float2 (&S)[NS / 2],
                                          float2 (&rate)[NS / 2]) {
#pragma unroll
    for (int i = 0; i < NS / 2; ++i) {
        float s[2] = {0.f, 0.f}, r[2] = {0.f, 0.f};
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const int n = n0 + 2 * i + k;
            if (live && n < a.states) {
                s[k] = st[(size_t)ch * a.states + n];
                r[k] = a.a[(size_t)ch * a.states + n] * RATE_UNIT<TA>;
            }
        }
        S[i] = make_float2(s[0], s[1]);
        rate[i] = make_float2(r[0], r[1]);
    }
}
template <int NS>
__device__ __forceinline__ void store_lane(const ScanArgs& a, float* st, int ch, int n0, bool live, const float2 (&S)[NS / 2]) {
#pragma unroll
    for (int i = 0; i < NS / 2; ++i) {
        const int n = n0 + 2 * i;
        if (live && n < a.states) st[(size_t)ch * a.states + n] = S[i].x;
        if (live && n + 1 < a.states) st[(size_t)ch * a.states + n + 1] = S[i].y;
    }
}

// A copy of N bytes (4 or 8) from global to shared memory that is waited for by group; zeros where !there.
template <int N> __device__ __forceinline__ void copy_async(void* dst, const void* src, bool there) {
    const int bytes = there ? N : 0;
    asm volatile("cp.async.ca.shared.global [%0], [%1], %2, %3;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src), "n"(N), "r"(bytes));
}
__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

template <int NS, int L> constexpr int STAGE = NS * L <= 64 ? 32 : 16;          // tokens of a stage
template <int L> constexpr int CHANNELS = WARPS * 32 / L;                        // channels of a block
template <int NS, int L> constexpr size_t KEYED_BYTES = (size_t)STAGE<NS, L> * NS * L * 2 * sizeof(float);
template <int L> constexpr int OUT_ROW = CHANNELS<L> + 4;      // four lanes' tokens lie in different banks
template <int NS, int L> constexpr size_t ROW_BYTES = (size_t)STAGE<NS, L> * (2 * CHANNELS<L> + OUT_ROW<L>) * sizeof(float);
template <int NS, int L> constexpr size_t SMEM = 3 * KEYED_BYTES<NS, L> + 2 * ROW_BYTES<NS, L>;

// W: values a bringing thread moves at once (4 where sizes and addresses allow it, else 1).
template <typename TA, int NS, int L, int W>
__global__ void __launch_bounds__(THREADS, NS == 2 ? 2 : 1)
selective_walk_kernel(const ScanArgs a) {
    constexpr int TS = STAGE<NS, L>, CB = CHANNELS<L>, NP = NS * L, CW = 32 / L;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int seg = blockIdx.y, q0 = a.seg_q_start[seg], n_tok = a.seg_q_start[seg + 1] - q0;
    if (n_tok <= 0) return;
    const int block_ch = blockIdx.x * CB, tid = threadIdx.x;
    const int stages = (n_tok + TS - 1) / TS;
    // a token's B and C: pair i as (b, b, c, c); then (step, step * x) an element; the walk's sums
    auto keyed_of = [&](int s) { return reinterpret_cast<float*>(smem_raw + (s % 3) * KEYED_BYTES<NS, L>); };
    auto steps_of = [&](int s) { return reinterpret_cast<float2*>(smem_raw + 3 * KEYED_BYTES<NS, L> + (s & 1) * ROW_BYTES<NS, L>); };
    auto sums_of = [&](int s) { return reinterpret_cast<float*>(steps_of(s) + TS * CB); };

    if (tid < ROLE) {
        // ------------------------------------------------------------------------------ the walk
        const int lane = tid & 31, l = lane % L, my = (tid >> 5) * CW + lane / L, ch = block_ch + my;
        const bool live = ch < a.inner, odd = l & 1, high = l & 2;
        float* st = a.state + (size_t)a.seg_slot[seg] * a.inner * a.states;
        float2 S[NS / 2], rate[NS / 2];
        load_lane<TA, NS>(a, st, ch, l * NS, live, S, rate);
        stage_barrier();                                // the first stage is there
        for (int s = 0; s < stages; ++s) {
            const int m = min(TS, n_tok - s * TS);
            const float2* steps = steps_of(s) + my;
            const float4* keyed = reinterpret_cast<const float4*>(keyed_of(s)) + l * (NS / 2);
            float* sums = sums_of(s) + my + (l & 3) * OUT_ROW<L>;
            // four tokens at a time, the rows of the next four and their decays asked for before this four's
            // read-outs are exchanged (at the stage's end the last four again, unused)
            float2 b[4][NS / 2], c[4][NS / 2], d[4][NS / 2];
            float input[4];
            auto rows_at = [&](int t0) {
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float2 step = steps[(t0 + j) * CB];
                    input[j] = step.y;
#pragma unroll
                    for (int i = 0; i < NS / 2; ++i) {
                        const float4 v = keyed[(t0 + j) * (NP / 2) + i];
                        b[j][i] = make_float2(v.x, v.y);
                        c[j][i] = make_float2(v.z, v.w);
                    }
                    decays<TA, NS>(d[j], rate, step.x);
                }
            };
            rows_at(0);
#pragma unroll 1
            for (int t0 = 0; t0 < m; t0 += 4) {
                float p[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) p[j] = advance<TA, NS>(S, d[j], input[j], b[j], c[j]);
                rows_at(min(t0 + 4, TS - 4));
                const float r0 = (odd ? p[1] : p[0]) + __shfl_xor_sync(0xffffffffu, odd ? p[0] : p[1], 1);
                const float r1 = (odd ? p[3] : p[2]) + __shfl_xor_sync(0xffffffffu, odd ? p[2] : p[3], 1);
                float q = (high ? r1 : r0) + __shfl_xor_sync(0xffffffffu, high ? r0 : r1, 2);
#pragma unroll
                for (int o = 4; o < L; o <<= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
                if (l < 4) sums[t0 * OUT_ROW<L>] = q;
            }
            stage_barrier();
        }
        store_lane<NS>(a, st, ch, l * NS, live, S);
        return;
    }
    // ------------------------------------------------------------------ bringing and carrying away
    const int me = tid - ROLE;
    constexpr int A_ROW = CB / W, ITEMS = (TS * A_ROW + ROLE - 1) / ROLE, ITEM_ROWS = ROLE / A_ROW;
    static_assert(ROLE % A_ROW == 0, "a bringing thread's items belong to the same channels");
    const int t_first = me / A_ROW, c = (me % A_ROW) * W, ch = block_ch + c;      // item i: token t_first + i * ITEM_ROWS
    const bool mine = ch < a.inner;                     // (W = 4: inner is a multiple of 4)
    const TA *x = (const TA*)a.x + (size_t)(q0 + t_first) * a.ldx + ch, *z = (const TA*)a.z + (size_t)(q0 + t_first) * a.ldz + ch;
    const float* dt = a.dt + (size_t)(q0 + t_first) * a.lddt + ch;
    // B and C: copies of a pair where a pair lies on 8 bytes (W = 4), else of an element
    constexpr int P = W == 4 ? 2 : 1, A_KEYED = NP / P, KEYED_ROWS = ROLE / A_KEYED, COPIES = (TS + KEYED_ROWS - 1) / KEYED_ROWS;
    static_assert(ROLE % A_KEYED == 0, "a bringing thread's copies belong to the same states");
    const int keyed_t = me / A_KEYED, keyed_n = (me % A_KEYED) * P, keyed_at = (keyed_t * NP + (keyed_n & ~1)) * 2 + (keyed_n & 1);
    const bool keyed_mine = keyed_n < a.states;         // (W = 4: the states are even)
    const size_t keyed_from = keyed_mine ? (size_t)min(keyed_t, n_tok - 1) * a.ldbc + keyed_n : 0;
    const float *bg = (const float*)a.b + (size_t)q0 * a.ldbc + keyed_from, *cg = (const float*)a.c + (size_t)q0 * a.ldbc + keyed_from;
    TA* out = (TA*)a.out + (size_t)(q0 + t_first) * a.ldo + ch;
    float bias[W], skip[W];
#pragma unroll
    for (int k = 0; k < W; ++k) {
        bias[k] = mine ? a.dt_bias[ch + k] : 0.f;
        skip[k] = mine ? a.skip[ch + k] : 0.f;
    }
    struct Rows {                                       // of one stage, as they lie in memory
        Piece<TA, W> x[ITEMS], z[ITEMS];
        Piece<float, W> dt[ITEMS];
        float2 end[ITEMS][W];                           // (skip * x, SiLU(z)) of the stage settled last
    } even, odd;
    auto fetch = [&](int s, Rows& held) {
        if (s < stages) {
            const int left = n_tok - s * TS;
#pragma unroll
            for (int i = 0; i < ITEMS; ++i) {
                const int t = t_first + i * ITEM_ROWS;
                if (mine && t < TS && t < left) {
                    const size_t row = (size_t)(s * TS + i * ITEM_ROWS);
                    held.x[i].load(x + row * a.ldx);
                    held.z[i].load(z + row * a.ldz);
                    held.dt[i].load(dt + row * a.lddt);
                }
            }
            float* to = keyed_of(s) + keyed_at;
#pragma unroll
            for (int i = 0; i < COPIES; ++i) {
                const int t = keyed_t + i * KEYED_ROWS;
                if (t >= TS) break;
                const bool there = keyed_mine && t < left;
                const long from = there ? (long)(s * TS + i * KEYED_ROWS) * a.ldbc : 0;
                copy_async<P * 4>(to + i * KEYED_ROWS * NP * 2, bg + from, there);
                copy_async<P * 4>(to + i * KEYED_ROWS * NP * 2 + 2, cg + from, there);
            }
        }
        copies_commit();                                // one group a stage, also an empty one
    };
    auto settle = [&](int s, Rows& held) {
        if (s >= stages) return;
        const int left = n_tok - s * TS;
#pragma unroll
        for (int i = 0; i < ITEMS; ++i) {
            const int t = t_first + i * ITEM_ROWS;
            if (t >= TS) continue;
            float2 step[W];
            if (mine && t < left) {
#pragma unroll
                for (int k = 0; k < W; ++k) {
                    const float v = to_float(held.x[i].v[k]);
                    step[k].x = softplus_f<TA>(held.dt[i].v[k] + bias[k]);
                    step[k].y = step[k].x * v;
                    held.end[i][k] = make_float2(__fmul_rn(skip[k], v), silu_f<TA>(to_float(held.z[i].v[k])));
                }
            } else {
#pragma unroll
                for (int k = 0; k < W; ++k) step[k] = make_float2(0.f, 0.f);
            }
            float2* to = steps_of(s) + t * CB + c;
            if constexpr (W == 4) {
#pragma unroll
                for (int k = 0; k < 4; k += 2)
                    *reinterpret_cast<float4*>(to + k) = make_float4(step[k].x, step[k].y, step[k + 1].x, step[k + 1].y);
            } else {
                to[0] = step[0];
            }
        }
    };
    auto carry = [&](int s, const Rows& held) {          // held: what stage s was settled from
        const int left = n_tok - s * TS;
#pragma unroll
        for (int i = 0; i < ITEMS; ++i) {
            const int t = t_first + i * ITEM_ROWS;
            if (mine && t < TS && t < left) {
                Piece<float, W> sum;
                Piece<TA, W> row;
                sum.load(sums_of(s) + t * OUT_ROW<L> + c);
#pragma unroll
                for (int k = 0; k < W; ++k) row.v[k] = from_float<TA>((sum.v[k] + held.end[i][k].x) * held.end[i][k].y);
                row.store(out + (size_t)(s * TS + i * ITEM_ROWS) * a.ldo);
            }
        }
    };
    // at a stage's barrier its successor's rows are formed and its copies have landed (all but the youngest group)
    fetch(0, even);
    fetch(1, odd);
    settle(0, even);
    copies_wait<1>();
    stage_barrier();
    for (int s = 0; s < stages; s += 2) {               // (the areas written here were walked before the last barrier)
        if (s > 0) carry(s - 1, odd);
        fetch(s + 2, even);
        settle(s + 1, odd);
        copies_wait<1>();
        stage_barrier();
        if (s + 1 == stages) break;
        carry(s, even);
        fetch(s + 3, odd);
        settle(s + 2, even);
        copies_wait<1>();
        stage_barrier();
    }
    if (stages & 1) carry(stages - 1, even);
    else carry(stages - 1, odd);
}

// A step in which every segment is a single token (or none).
template <typename TA, int NS, int L>
__global__ void __launch_bounds__(SINGLE)
selective_single_kernel(const ScanArgs a) {
    const int seg = blockIdx.y, q0 = a.seg_q_start[seg];
    if (a.seg_q_start[seg + 1] <= q0) return;
    const int lane = threadIdx.x & 31, l = lane % L, ch = (blockIdx.x * SINGLE + threadIdx.x) / L;
    const bool live = ch < a.inner;
    float* st = a.state + (size_t)a.seg_slot[seg] * a.inner * a.states;
    float2 S[NS / 2], rate[NS / 2], b[NS / 2], c[NS / 2];
    load_lane<TA, NS>(a, st, ch, l * NS, live, S, rate);
    const TA *bg = (const TA*)a.b + (size_t)q0 * a.ldbc, *cg = (const TA*)a.c + (size_t)q0 * a.ldbc;
#pragma unroll
    for (int i = 0; i < NS / 2; ++i) {
        const int n = l * NS + 2 * i;
        b[i] = make_float2(n < a.states ? to_float(bg[n]) : 0.f, n + 1 < a.states ? to_float(bg[n + 1]) : 0.f);
        c[i] = make_float2(n < a.states ? to_float(cg[n]) : 0.f, n + 1 < a.states ? to_float(cg[n + 1]) : 0.f);
    }
    float step = 0.f, v = 0.f;
    if (live) {
        v = to_float(((const TA*)a.x)[(size_t)q0 * a.ldx + ch]);
        step = softplus_f<TA>(a.dt[(size_t)q0 * a.lddt + ch] + a.dt_bias[ch]);
    }
    float2 d[NS / 2];
    decays<TA, NS>(d, rate, step);
    float q = advance<TA, NS>(S, d, step * v, b, c);
#pragma unroll
    for (int o = 1; o < L; o <<= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
    store_lane<NS>(a, st, ch, l * NS, live, S);
    if (live && l == 0)
        ((TA*)a.out)[(size_t)q0 * a.ldo + ch] =
            from_float<TA>((q + __fmul_rn(a.skip[ch], v)) * silu_f<TA>(to_float(((const TA*)a.z)[(size_t)q0 * a.ldz + ch])));
}

template <typename TA, int NS, int L>
int launch(const ScanArgs& a, int segments, int max_q_len, cudaStream_t stream) {
    if (max_q_len == 1) {
        constexpr int PER = SINGLE / L;
        selective_single_kernel<TA, NS, L><<<dim3((a.inner + PER - 1) / PER, segments), SINGLE, 0, stream>>>(a);
        MRUN_CHECK_LAUNCH("selective_scan");
        return 0;
    }
    constexpr size_t smem = SMEM<NS, L>, unit = 4 * sizeof(TA);
    static_assert(smem <= 110 * 1024, "two blocks' stages must fit a multiprocessor's shared memory");
    const dim3 grid((a.inner + CHANNELS<L> - 1) / CHANNELS<L>, segments);
    auto on = [&](const void* p, long ld, size_t bytes) { return (uintptr_t)p % bytes == 0 && ld % 4 == 0; };
    const bool wide = a.inner % 4 == 0 && a.states % 2 == 0 && on(a.x, a.ldx, unit) && on(a.z, a.ldz, unit) && on(a.b, a.ldbc, 8) &&
                      on(a.c, a.ldbc, 8) && on(a.out, a.ldo, unit) && on(a.dt, a.lddt, 16);
    auto start = [&](void (*kernel)(const ScanArgs)) {
        if (smem > 48 * 1024)
            MRUN_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem), "selective_scan");
        kernel<<<grid, THREADS, smem, stream>>>(a);
        MRUN_CHECK_LAUNCH("selective_scan");
        return 0;
    };
    return wide ? start(selective_walk_kernel<TA, NS, L, 4>) : start(selective_walk_kernel<TA, NS, L, 1>);
}

template <typename TA>
int dispatch(const ScanArgs& a, int segments, int max_q_len, cudaStream_t stream) {
    const int n = a.states;
    if (n <= 8) return launch<TA, 2, 4>(a, segments, max_q_len, stream);
    if (n <= 16) return launch<TA, 2, 8>(a, segments, max_q_len, stream);
    if (n <= 32) return launch<TA, 2, 16>(a, segments, max_q_len, stream);
    if (n <= 64) return launch<TA, 2, 32>(a, segments, max_q_len, stream);
    if (n <= 128) return launch<TA, 4, 32>(a, segments, max_q_len, stream);
    return launch<TA, 8, 32>(a, segments, max_q_len, stream);
}

}  // namespace

// x, z: [tokens, inner] of the activation type; b, c: [tokens, states] of 32-bit floats, of the activation type
// where max_q_len is 1 (a step of single tokens); rows with the given strides.  dt: float32 [tokens, inner], the step before its bias and softplus.  a: float32 [inner, states], the
// (negative) rates.  state: float32 [slots, inner, states].
MRUN_API int mrun_selective_scan(const void* x, long ldx, const void* z, long ldz, const void* b, const void* c, long ldbc,
                                 int act_dtype, const float* dt, long lddt, const float* dt_bias, const float* a,
                                 const float* skip, float* state, void* out, long ldo, const int* seg_q_start,
                                 const int* seg_slot, int segments, int max_q_len, int tokens, int inner, int states,
                                 cudaStream_t stream) {
    MRUN_REQUIRE(tokens >= 0 && segments >= 0 && segments <= 65535 && inner > 0 && states > 0,
                 "selective_scan: bad sizes tokens=%d segments=%d inner=%d states=%d", tokens, segments, inner, states);
    MRUN_REQUIRE(states <= 256, "selective_scan: %d states a channel exceed the supported 256", states);
    MRUN_REQUIRE(ldx >= inner && ldz >= inner && ldbc >= states && lddt >= inner && ldo >= inner,
                 "selective_scan: a row stride is below the row");
    if (tokens == 0 || segments == 0) return 0;
    const ScanArgs args = {x, z, b, c, ldx, ldz, ldbc, dt, lddt, dt_bias, a, skip, state, out, ldo, seg_q_start, seg_slot, inner, states};
    if (act_dtype == MRUN_F32) return dispatch<float>(args, segments, max_q_len, stream);
    if (act_dtype == MRUN_BF16) return dispatch<__nv_bfloat16>(args, segments, max_q_len, stream);
    return mrun_set_error("selective_scan: unknown dtype code %d", act_dtype);
}
