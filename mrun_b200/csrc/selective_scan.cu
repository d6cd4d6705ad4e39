// The selective scan of a state-space mixer whose decays belong to channels and states (Mamba): per
// request, channel c and state n, over the request's tokens,
//
//   step_c = softplus(dt_c + bias_c)
//   S[c, n] <- exp(step_c A[c, n]) S[c, n] + step_c x_c B_n
//   out_c   = (sum_n S[c, n] C_n + skip_c x_c) * SiLU(z_c)
//
// from and into the request's state (float32 [inner, states]).  Everything but the rows themselves is 32-bit.
//
// A lane holds NS states of one channel as pairs (packed 32-bit arithmetic), L lanes hold a channel.  Four
// warps of a block walk; four others bring the input of the stage ahead (steps, step * x, skip * x and
// SiLU(z) formed once an element, B and C widened) and carry the finished rows of the stage behind to
// memory.  The roles meet at one barrier a stage; stages are double-buffered in shared memory.
//
// A walking lane's bound is the exponential, one a state and token; so four tokens go side by side and their
// read-outs are summed over the channel's lanes together: two exchanges halve the tokens a lane is in
// charge of, so that lane l of the first four ends with token l's sum (three shuffles for four tokens).
// The sum of a token is ((l0 + l1) + (l2 + l3)) + ... whatever its place, a step without a token has step 0
// and leaves the state as it is (decay 1, nothing written), so a token's result has the same bits however its request was
// cut.  A step of single tokens has a smaller kernel with the same arithmetic.
// grid: channel groups x segments; a segment of zero rows is padding.
#include "common.cuh"

using namespace mrun;

namespace {

constexpr int WARPS = 4;                    // of each of the two roles
constexpr int ROLE = WARPS * 32, THREADS = 2 * ROLE;

struct ScanArgs {
    const void *x, *z, *b, *c;              // rows of the activation type
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

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ void stage_barrier() { asm volatile("bar.sync 1, %0;" ::"n"(THREADS) : "memory"); }
__device__ __forceinline__ float2 both(float v) { return make_float2(v, v); }
__device__ __forceinline__ float exp2_fast(float v) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
    return r;
}
// What a decay's rate is multiplied by when it is loaded: the 16-bit path takes powers of two.
template <typename TA> constexpr float RATE_UNIT = sizeof(TA) == 4 ? 1.f : 1.4426950408889634f;

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

// One token of a lane's states: they advance, the lane's share of the read-out comes back.
template <typename TA, int NS>
__device__ __forceinline__ float advance(float2 (&S)[NS / 2], const float2 (&rate)[NS / 2], float step, float input,
                                         const float2 (&b)[NS / 2], const float2 (&c)[NS / 2]) {
    float2 acc = both(0.f);
#pragma unroll
    for (int i = 0; i < NS / 2; ++i) {
        const float2 arg = __fmul2_rn(both(step), rate[i]), write = __fmul2_rn(both(input), b[i]);
        if constexpr (sizeof(TA) == 4) {        // S + ((decay - 1) S + write): a decay next to one keeps its digits
            const float2 loss = make_float2(expm1f(arg.x), expm1f(arg.y));
            S[i] = __fadd2_rn(S[i], __ffma2_rn(loss, S[i], write));
        } else {
            S[i] = __ffma2_rn(make_float2(exp2_fast(arg.x), exp2_fast(arg.y)), S[i], write);
        }
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

template <int NS, int L> constexpr int STAGE = NS * L <= 64 ? 32 : 16;          // tokens of a stage
template <int L> constexpr int CHANNELS = WARPS * 32 / L;                        // channels of a block
template <typename TA, int NS, int L> constexpr size_t BUFFER = (size_t)STAGE<NS, L> * (CHANNELS<L> * (4 * sizeof(float) + sizeof(TA)) + 2 * NS * L * sizeof(float));

// W: values a bringing thread moves at once (4 where sizes and addresses allow it, else 1).
template <typename TA, int NS, int L, int W>
__global__ void __launch_bounds__(THREADS)
selective_walk_kernel(const ScanArgs a) {
    constexpr int TS = STAGE<NS, L>, CB = CHANNELS<L>, NP = NS * L, CW = 32 / L;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int seg = blockIdx.y, q0 = a.seg_q_start[seg], n_tok = a.seg_q_start[seg + 1] - q0;
    if (n_tok <= 0) return;
    const int block_ch = blockIdx.x * CB, tid = threadIdx.x;
    const int stages = (n_tok + TS - 1) / TS;
    // a stage's area: (step, step * x) and (skip * x, SiLU(z)) an element, B and C rows, finished rows
    auto steps_of = [&](int s) { return reinterpret_cast<float2*>(smem_raw + (s & 1) * BUFFER<TA, NS, L>); };
    auto ends_of = [&](int s) { return steps_of(s) + TS * CB; };
    auto b_of = [&](int s) { return reinterpret_cast<float*>(ends_of(s) + TS * CB); };
    auto c_of = [&](int s) { return b_of(s) + TS * NP; };
    auto out_of = [&](int s) { return reinterpret_cast<TA*>(c_of(s) + TS * NP); };

    if (tid < ROLE) {
        // ------------------------------------------------------------------------------ the walk
        const int lane = tid & 31, l = lane % L, my = (tid >> 5) * CW + lane / L, ch = block_ch + my;
        const bool live = ch < a.inner;
        float* st = a.state + (size_t)a.seg_slot[seg] * a.inner * a.states;
        float2 S[NS / 2], rate[NS / 2];
        load_lane<TA, NS>(a, st, ch, l * NS, live, S, rate);
        stage_barrier();                                // the first stage is there
        for (int s = 0; s < stages; ++s) {
            const int m = min(TS, n_tok - s * TS);
            const float2 *steps = steps_of(s) + my, *ends = ends_of(s) + my;
            const float *bs = b_of(s) + l * NS, *cs = c_of(s) + l * NS;
            TA* rows = out_of(s) + my;
            for (int t0 = 0; t0 < m; t0 += 4) {
                float p[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int t = t0 + j;
                    const float2 step = steps[t * CB];
                    float2 b[NS / 2], c[NS / 2];
#pragma unroll
                    for (int i = 0; i < NS / 2; ++i) {
                        b[i] = *reinterpret_cast<const float2*>(bs + t * NP + 2 * i);
                        c[i] = *reinterpret_cast<const float2*>(cs + t * NP + 2 * i);
                    }
                    p[j] = advance<TA, NS>(S, rate, step.x, step.y, b, c);
                }
                const bool odd = l & 1, high = l & 2;
                const float r0 = (odd ? p[1] : p[0]) + __shfl_xor_sync(0xffffffffu, odd ? p[0] : p[1], 1);
                const float r1 = (odd ? p[3] : p[2]) + __shfl_xor_sync(0xffffffffu, odd ? p[2] : p[3], 1);
                float q = (high ? r1 : r0) + __shfl_xor_sync(0xffffffffu, high ? r0 : r1, 2);
#pragma unroll
                for (int o = 4; o < L; o <<= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
                if (l < 4) {
                    const float2 end = ends[(t0 + l) * CB];
                    rows[(t0 + l) * CB] = from_float<TA>((q + end.x) * end.y);
                }
            }
            stage_barrier();
        }
        store_lane<NS>(a, st, ch, l * NS, live, S);
        return;
    }
    // ------------------------------------------------------------------ bringing and carrying away
    const int me = tid - ROLE;
    constexpr int ITEMS = (TS * CB / W + ROLE - 1) / ROLE;
    const TA *x = (const TA*)a.x + (size_t)q0 * a.ldx, *z = (const TA*)a.z + (size_t)q0 * a.ldz;
    const TA *bg = (const TA*)a.b + (size_t)q0 * a.ldbc, *cg = (const TA*)a.c + (size_t)q0 * a.ldbc;
    const float* dt = a.dt + (size_t)q0 * a.lddt;
    TA* out = (TA*)a.out + (size_t)q0 * a.ldo;
    Piece<TA, W> xs[ITEMS], zs[ITEMS];
    Piece<float, W> ds[ITEMS];
    auto place = [&](int i, int& t, int& c) {           // item i of this thread: token and first channel
        const int e = me + i * ROLE;
        t = e / (CB / W);
        c = (e - t * (CB / W)) * W;
    };
    auto fetch = [&](int s) {
        const int m = min(TS, n_tok - s * TS);
#pragma unroll
        for (int i = 0; i < ITEMS; ++i) {
            int t, c;
            place(i, t, c);
            if (t < m && block_ch + c < a.inner) {      // (W = 4: inner is a multiple of 4)
                const size_t row = (size_t)(s * TS + t);
                xs[i].load(x + row * a.ldx + block_ch + c);
                zs[i].load(z + row * a.ldz + block_ch + c);
                ds[i].load(dt + row * a.lddt + block_ch + c);
            }
        }
        // B and C are widened at once: their latency is hidden by what follows only in part
        const int whole = (m + 3) & ~3;
        for (int e = me; e < whole * (NP / W); e += ROLE) {
            const int t = e / (NP / W), n = (e - t * (NP / W)) * W;
            Piece<TA, W> pb, pc;
            const bool there = t < m && n < a.states;   // (W = 4: the states are a multiple of 4)
            if (there) {
                pb.load(bg + (size_t)(s * TS + t) * a.ldbc + n);
                pc.load(cg + (size_t)(s * TS + t) * a.ldbc + n);
            }
#pragma unroll
            for (int k = 0; k < W; ++k) {
                b_of(s)[t * NP + n + k] = there ? to_float(pb.v[k]) : 0.f;
                c_of(s)[t * NP + n + k] = there ? to_float(pc.v[k]) : 0.f;
            }
        }
    };
    auto settle = [&](int s) {
        const int m = min(TS, n_tok - s * TS);
#pragma unroll
        for (int i = 0; i < ITEMS; ++i) {
            int t, c;
            place(i, t, c);
            if (t >= TS) continue;
            const bool there = t < m && block_ch + c < a.inner;
#pragma unroll
            for (int k = 0; k < W; ++k) {
                float2 step = make_float2(0.f, 0.f), end = make_float2(0.f, 0.f);
                if (there) {
                    const int ch = block_ch + c + k;
                    const float v = to_float(xs[i].v[k]);
                    step.x = softplus_f(ds[i].v[k] + a.dt_bias[ch]);
                    step.y = step.x * v;
                    end = make_float2(__fmul_rn(a.skip[ch], v), silu_f(to_float(zs[i].v[k])));
                }
                steps_of(s)[t * CB + c + k] = step;
                ends_of(s)[t * CB + c + k] = end;
            }
        }
    };
    auto carry = [&](int s) {
        const int m = min(TS, n_tok - s * TS);
#pragma unroll
        for (int i = 0; i < ITEMS; ++i) {
            int t, c;
            place(i, t, c);
            if (t < m && block_ch + c < a.inner) {
                Piece<TA, W> row;
                row.load(out_of(s) + t * CB + c);
                row.store(out + (size_t)(s * TS + t) * a.ldo + block_ch + c);
            }
        }
    };
    fetch(0);
    settle(0);
    stage_barrier();
    for (int s = 0; s < stages; ++s) {
        if (s + 1 < stages) fetch(s + 1);
        if (s > 0) carry(s - 1);
        if (s + 1 < stages) settle(s + 1);
        stage_barrier();
    }
    carry(stages - 1);
}

// A step in which every segment is a single token (or none).
template <typename TA, int NS, int L>
__global__ void __launch_bounds__(ROLE)
selective_single_kernel(const ScanArgs a) {
    const int seg = blockIdx.y, q0 = a.seg_q_start[seg];
    if (a.seg_q_start[seg + 1] <= q0) return;
    const int lane = threadIdx.x & 31, l = lane % L, ch = (blockIdx.x * ROLE + threadIdx.x) / L;
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
        step = softplus_f(a.dt[(size_t)q0 * a.lddt + ch] + a.dt_bias[ch]);
    }
    float q = advance<TA, NS>(S, rate, step, step * v, b, c);
#pragma unroll
    for (int o = 1; o < L; o <<= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
    store_lane<NS>(a, st, ch, l * NS, live, S);
    if (live && l == 0)
        ((TA*)a.out)[(size_t)q0 * a.ldo + ch] =
            from_float<TA>((q + __fmul_rn(a.skip[ch], v)) * silu_f(to_float(((const TA*)a.z)[(size_t)q0 * a.ldz + ch])));
}

template <typename TA, int NS, int L>
int launch(const ScanArgs& a, int segments, int max_q_len, cudaStream_t stream) {
    if (max_q_len == 1) {
        constexpr int PER = ROLE / L;
        selective_single_kernel<TA, NS, L><<<dim3((a.inner + PER - 1) / PER, segments), ROLE, 0, stream>>>(a);
        MRUN_CHECK_LAUNCH("selective_scan");
        return 0;
    }
    constexpr size_t smem = 2 * BUFFER<TA, NS, L>, unit = 4 * sizeof(TA);
    static_assert(smem <= 200 * 1024, "the stages must fit a block's shared memory");
    const dim3 grid((a.inner + CHANNELS<L> - 1) / CHANNELS<L>, segments);
    auto on = [&](const void* p, long ld) { return (uintptr_t)p % unit == 0 && ld % 4 == 0; };
    const bool wide = a.inner % 4 == 0 && a.states % 4 == 0 && on(a.x, a.ldx) && on(a.z, a.ldz) && on(a.b, a.ldbc) &&
                      on(a.c, a.ldbc) && on(a.out, a.ldo) && (uintptr_t)a.dt % 16 == 0 && a.lddt % 4 == 0;
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
    if (n <= 16) return launch<TA, 4, 4>(a, segments, max_q_len, stream);
    if (n <= 32) return launch<TA, 4, 8>(a, segments, max_q_len, stream);
    if (n <= 64) return launch<TA, 4, 16>(a, segments, max_q_len, stream);
    if (n <= 128) return launch<TA, 4, 32>(a, segments, max_q_len, stream);
    return launch<TA, 8, 32>(a, segments, max_q_len, stream);
}

}  // namespace

// x, z: [tokens, inner]; b, c: [tokens, states]; rows of the activation type with the given strides.  dt:
// float32 [tokens, inner], the step before its bias and softplus.  a: float32 [inner, states], the
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
