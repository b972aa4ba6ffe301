// Walks over matrix states that take a request's tokens eight at a time, over a flat batch of requests (each brings a prompt's
// portion or one decoded token). Per head a state S [key channel x value channel] of 32-bit floats, in a slot of a state tensor
// (row stride `state_ld`, from column `state_off`, laid out [head, value channel, key channel]); which request owns which rows
// and which slot is read from device arrays, so a captured graph can replay the launches for other requests. Two rules, all
// arithmetic 32-bit:
//
//   delta:   S <- diag(w_t) S,   u_t = beta_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   o_t = S^T q_t
//   plain:   S <- diag(w_t) S + k_t v_t^T,                                             o_t = S^T q_t
//
// Within a group of GS_T tokens everything that does not involve S can be known before S is. With W_t the product of the
// group's decays up to and including token t, and W_(s,t] the product of those after s up to t,
//
//     u_t = beta_t (v_t - (W_t k_t)^T S_0 - sum_(s<t) c_ts u_s),     c_ts = sum_ch k_t k_s W_(s,t],
//     o_t = (W_t q_t)^T S_0 + sum_(s<=t) d_ts u_s,                   d_ts = sum_ch q_t k_s W_(s,t],
//     S_n = W_n S_0 + sum_s (W_(s,n] k_s) u_s^T                      (plain: u = v)
//
// so for the delta rule u = A (v - (W k)^T S_0) with A = (I + diag(beta) C)^(-1) diag(beta), a lower triangular matrix per
// (group, head) that all value channels share. Only products of decays appear (no quotients), so strong decays underflow to
// zero harmlessly.
//  * group_prepare: a warp per (group, head): unit keys and queries, decays, beta, the vectors W_t k_t, W_t q_t, W_(s,n] k_s,
//    W_n, and the matrices A and D; parallel over the whole step.
//    What the walk reads of a (group, head) lies in ONE block of the scratch.
//  * state_step: steps in which no request brings more than GS_STEP_TOKENS tokens (a decode step): the rules as they stand, token by
//    token, in one launch; a warp per GS_STEP_COLS value channels of a head of a request, every warp forming what it needs of q, k,
//    the decays and beta by itself.
//  * group_walk: a warp per one or two value channels of a head of a request, their key channels in the lanes' registers (two
//    channels read a staged vector once: where the walk is bound by shared memory, not by its chain); the warps of a block
//    share a group's block, which a warp of its own brings into shared memory (one bulk copy) several groups ahead. Per group: dot products with S_0 for the eight tokens, their sums over the lanes together (each
//    exchange halves what a lane holds), 8 x 8 products with the matrices, one update of S.
// Groups start at the step's first token of a request: a result depends on how the request was cut by rounding only.
#include "pipeline.cuh"
#include <type_traits>

using namespace nibp;

constexpr int GS_T = 8;             // tokens per group
constexpr int GS_STEP_TOKENS = 4, GS_STEP_COLS = 4;     // short steps: tokens per request at most, value channels per warp

__device__ int g_group_walk_error = 0;      // 0, or (role << 16 | blockIdx.x) of the first wait that ran out (1 a walking warp, 2 the sending one)

// A (group, head)'s block, in floats: W_t q_t, W_(t,n] k_t and (delta) W_t k_t for the eight tokens (rows of DKP floats, channels
// beyond dk and tokens that do not exist zero), W_n, D and (delta) A.
template <int C, bool DELTA> struct GsLayout {
    static constexpr int NC = C >= 8 || (DELTA && C < 4) ? 1 : 2;           // value channels per warp
    static constexpr int WARPS = 4, COLS = WARPS * NC;         // walking warps, value channels per block of threads
    static constexpr int DKP = 32 * C, VECS = DELTA ? 3 : 2;
    static constexpr int Q0 = 0, S0 = GS_T * DKP, K0 = 2 * GS_T * DKP, W0 = VECS * GS_T * DKP, D0 = W0 + DKP, A0 = D0 + GS_T * GS_T,
                         SIZE = A0 + (DELTA ? GS_T * GS_T : 0);
    static constexpr int STAGES = C >= 8 ? 3 : 4;
    static constexpr int BYTES = STAGES * SIZE * 4;
};

// The block index of a request's first group: requests' groups lie one behind the other, with room for one group that is not
// full per request.
__device__ __forceinline__ long long first_group(int row0, int req) { return row0 / GS_T + req; }

// exp(x) for x <= 0 or a little above: near zero 1 + expm1, so that a result near one is off by its own rounding alone (a decay
// is raised to hundreds of powers along a sequence, which would multiply a bias of expf up).
__device__ __forceinline__ float gs_decay_exp(float x) { return fabsf(x) < 0.5f ? 1.0f + expm1f(x) : expf(x); }

// exp(-rate softplus(x))
__device__ __forceinline__ float gs_step_decay(float x, float rate) {
    return gs_decay_exp(-rate * (x > 0.f ? x + log1pf(expf(-x)) : log1pf(expf(x))));
}

// How z is read: GS_STEP per (head, key channel) logits of step sizes, decay = exp(-rate[h] * softplus(z + dt_bias));
// GS_CHANNEL per (head, key channel) decays; GS_HEAD one decay per head.
enum { GS_STEP = 0, GS_CHANNEL = 1, GS_HEAD = 2 };

template <int CPL, bool DELTA>
__global__ void __launch_bounds__(128)
group_prepare_kernel(const float* __restrict__ q, int ldq, const float* __restrict__ k, int ldk, const float* __restrict__ z, int ldz, int z_kind,
                     const float* __restrict__ dt_bias, const float* __restrict__ rate, const float* __restrict__ b, int ldb,
                     const float* __restrict__ k_scale, const int* __restrict__ q_start, float* __restrict__ work, int heads, int kq_heads, int dk,
                     float q_scale, float unit_eps) {
    pdl_launch_dependents();
    pdl_wait();      // everything this kernel reads may come from the kernel before
    __shared__ float s_m[4][GS_T * GS_T];       // per warp: D on and below the diagonal, C mirrored above it
    __shared__ float s_beta[4][GS_T];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, req = blockIdx.y;
    const int wid = blockIdx.x * 4 + warp;
    const int group = wid / heads, h = wid - group * heads;
    const int first = q_start[req], len = q_start[req + 1] - first;
    if (group * GS_T >= len) return;            // a whole warp leaves together, and nothing below waits for the block
    const int row0 = first + group * GS_T, nt = min(GS_T, len - group * GS_T);
    const int hq = h / (heads / kq_heads);
    using L = GsLayout<CPL, DELTA>;
    float* blk = work + ((first_group(first, req) + group) * heads + h) * L::SIZE;
    const float r = z_kind == GS_STEP ? rate[h] : 0.f;
    float bias[CPL];
#pragma unroll
    for (int i = 0; i < CPL; ++i) bias[i] = (z_kind == GS_STEP && lane + 32 * i < dk) ? dt_bias[(size_t)h * dk + lane + 32 * i] : 0.f;
    // everything the group reads is sent for at once
    float kv[GS_T][CPL], qv[GS_T][CPL], wv[GS_T][CPL];
#pragma unroll
    for (int t = 0; t < GS_T; ++t) {
        const bool on = t < nt;
        const size_t row = (size_t)(row0 + (on ? t : 0));
        const float wh = z_kind == GS_HEAD ? z[row * ldz + h] : 1.f;
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
            const int c = lane + 32 * i;
            const bool in = on && c < dk;
            kv[t][i] = in ? k[row * ldk + (size_t)hq * dk + c] : 0.f;
            qv[t][i] = in ? q[row * ldq + (size_t)hq * dk + c] : 0.f;
            wv[t][i] = !in ? 1.f : (z_kind == GS_HEAD ? wh : z[row * ldz + (size_t)h * dk + c]);
        }
    }
    if (DELTA && lane < nt) s_beta[warp][lane] = 1.0f / (1.0f + expf(-b[(size_t)(row0 + lane) * ldb + h]));
    float run[GS_T][CPL];       // k_s times the decays after s so far
    float pre[CPL];             // the product of the decays so far
    float acc[GS_T * GS_T];
#pragma unroll
    for (int i = 0; i < GS_T * GS_T; ++i) acc[i] = 0.f;
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
        pre[i] = 1.f;
#pragma unroll
        for (int s = 0; s < GS_T; ++s) run[s][i] = 0.f;
    }
#pragma unroll
    for (int t = 0; t < GS_T; ++t) {
        if (t >= nt) continue;
        const size_t row = (size_t)(row0 + t);
        float ik = 1.0f, iq = q_scale;
        if (unit_eps >= 0.f) {
            float sk = 0.f, sq = 0.f;
#pragma unroll
            for (int i = 0; i < CPL; ++i) { sk = fmaf(kv[t][i], kv[t][i], sk); sq = fmaf(qv[t][i], qv[t][i], sq); }
            ik = 1.0f / sqrtf(warp_sum(sk) + unit_eps);
            iq = q_scale / sqrtf(warp_sum(sq) + unit_eps);
        }
        if (k_scale != nullptr) ik *= k_scale[row * heads + h];
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
            const int c = lane + 32 * i;
            float w = wv[t][i];
            if (z_kind == GS_STEP && c < dk) w = gs_step_decay(w + bias[i], r);
            const float ku = kv[t][i] * ik, qu = qv[t][i] * iq;
            pre[i] *= w;
#pragma unroll
            for (int s = 0; s < GS_T; ++s) {
                if (s < t) {
                    run[s][i] *= w;
                    acc[t * GS_T + s] = fmaf(qu, run[s][i], acc[t * GS_T + s]);
                    if (DELTA) acc[s * GS_T + t] = fmaf(ku, run[s][i], acc[s * GS_T + t]);
                }
            }
            run[t][i] = ku;
            acc[t * GS_T + t] = fmaf(qu, ku, acc[t * GS_T + t]);
            if (DELTA) blk[L::K0 + t * L::DKP + c] = ku * pre[i];
            blk[L::Q0 + t * L::DKP + c] = qu * pre[i];
        }
    }
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
        const int c = lane + 32 * i;
#pragma unroll
        for (int s = 0; s < GS_T; ++s) {
            blk[L::S0 + s * L::DKP + c] = run[s][i];
            if (s >= nt) {      // tokens that do not exist
                if (DELTA) blk[L::K0 + s * L::DKP + c] = 0.f;
                blk[L::Q0 + s * L::DKP + c] = 0.f;
            }
        }
        blk[L::W0 + c] = pre[i];
    }
    // the 64 sums over the lanes together: five exchanges, each lane keeping half of what it held; lane l ends with the
    // sums 2 l and 2 l + 1
#pragma unroll
    for (int half = 32, o = 16; o > 0; half >>= 1, o >>= 1) {
        const bool up = (lane & o) != 0;
#pragma unroll
        for (int i = 0; i < 32; ++i) {
            if (i >= half) continue;
            const float recv = __shfl_xor_sync(0xffffffffu, up ? acc[i] : acc[i + half], o);
            acc[i] = (up ? acc[i + half] : acc[i]) + recv;
        }
    }
    float* m = s_m[warp];
    m[2 * lane] = acc[0];
    m[2 * lane + 1] = acc[1];
    __syncwarp();
    if (lane < GS_T) {
        // column `lane` of A by forward substitution: x_t = beta_t ([t == lane] - sum_(s<t) c_ts x_s); row `lane` of D
        if (DELTA) {
            float x[GS_T];
#pragma unroll
            for (int t = 0; t < GS_T; ++t) {
                float sum = t == lane ? 1.f : 0.f;
#pragma unroll
                for (int s = 0; s < GS_T; ++s)
                    if (s < t) sum = fmaf(-m[s * GS_T + t], x[s], sum);
                x[t] = t < nt ? s_beta[warp][t] * sum : 0.f;
                blk[L::A0 + t * GS_T + lane] = x[t];
            }
        }
        float* d = blk + L::D0 + lane * GS_T;
#pragma unroll
        for (int s = 0; s < GS_T; ++s) d[s] = (lane < nt && s <= lane) ? m[lane * GS_T + s] : 0.f;
    }
}

template <int C, bool DELTA>
__global__ void __launch_bounds__(GsLayout<C, DELTA>::WARPS * 32 + 32)
group_walk_kernel(const float* __restrict__ work, const float* __restrict__ v, int ldv, float* __restrict__ state, long long state_ld, int state_off,
                  const int* __restrict__ q_start, const int* __restrict__ slots, float* __restrict__ o, int ldo, int heads, int dk, int dv,
                  int ones) {
    using L = GsLayout<C, DELTA>;
    constexpr int DKP = L::DKP, STAGES = L::STAGES, WARPS = L::WARPS, NC = L::NC, COLS = L::COLS;
    extern __shared__ __align__(16) float gs_smem[];
    __shared__ unsigned long long full[STAGES], empty[STAGES];
    __shared__ __align__(16) float s_v[STAGES][COLS * GS_T];      // a channel's eight values lie together
    __shared__ volatile int s_failed;
    const int req = blockIdx.z, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int cols = dv + ones, j0 = blockIdx.x * COLS + warp * NC;      // value channels of the state, a column of ones behind the others
    const int row0 = q_start[req], row1 = q_start[req + 1];
    const int groups = (row1 - row0 + GS_T - 1) / GS_T;
    if (threadIdx.x == 0) {
        s_failed = 0;
        // full: the block's copy (its one arrival counts the bytes) and the 32 lanes' values; empty: one arrival per walking warp
        for (int i = 0; i < STAGES; ++i) { mbar_init(&full[i], 33); mbar_init(&empty[i], WARPS); }
        mbar_fence_init();
    }
    __syncthreads();
    pdl_wait();      // everything below may come from the kernels before
    const float* src = work + (first_group(row0, req) * heads + h) * L::SIZE;
    if (warp == WARPS) {        // ---------------- the warp that sends for the groups
        int sent = 0;
        for (int g = 0; g < groups && !s_failed; ++g) {
            const int st = g % STAGES;
            bool ok = true;
            if (g >= STAGES) ok = __all_sync(0xffffffffu, mbar_wait(&empty[st], (g / STAGES - 1) & 1));
            if (!ok) {
                if (lane == 0) atomicCAS(&g_group_walk_error, 0, (2 << 16) | (int)(blockIdx.x & 0xffff));
                s_failed = 1;
                break;
            }
            if (lane == 0) {
                mbar_expect_tx(&full[st], L::SIZE * 4);
                bulk_copy_g2s(gs_smem + st * L::SIZE, src + (size_t)g * heads * L::SIZE, L::SIZE * 4, &full[st]);
            }
#pragma unroll
            for (int e = lane; e < GS_T * COLS; e += 32) {     // the values of the block's channels (a column of ones has none)
                const int t = g * GS_T + e % GS_T, jj = blockIdx.x * COLS + e / GS_T;
                const bool there = t < row1 - row0 && jj < dv;
                const float* from = v + (size_t)(row0 + (there ? t : 0)) * ldv + (size_t)h * dv + (there ? jj : 0);
                const int n = there ? 4 : 0;        // 0 source bytes: the destination is zero-filled
                asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"(smem_u32(&s_v[st][e])), "l"(from), "r"(n));
            }
            asm volatile("cp.async.mbarrier.arrive.noinc.shared::cta.b64 [%0];\n" ::"r"(smem_u32(&full[st])) : "memory");
            sent = g + 1;
        }
        // nobody leaves with copies in flight: after a failure their arrival is waited for, bounded
        if (s_failed)
            for (int g = max(0, sent - STAGES); g < sent; ++g) mbar_wait(&full[g % STAGES], (g / STAGES) & 1);
        asm volatile("cp.async.wait_all;\n" ::: "memory");
        return;
    }
    float* head_state = state + (long long)slots[req] * state_ld + state_off + (long long)h * cols * dk;
    // lane l owns the channels l * C .. + C - 1 (C = 8: l * 4 .. + 3 of both halves): a warp's load of a vector is contiguous
    auto channel = [&](int i) { return C == 8 ? (i >> 2) * 128 + lane * 4 + (i & 3) : lane * C + i; };
    float S[NC][C];
#pragma unroll
    for (int n = 0; n < NC; ++n)
#pragma unroll
        for (int i = 0; i < C; ++i) S[n][i] = (j0 + n < cols && channel(i) < dk) ? head_state[(long long)(j0 + n) * dk + channel(i)] : 0.f;
    auto take = [&](const float* row, float (&x)[C]) {
        if constexpr (C == 1) x[0] = row[lane];
        else if constexpr (C == 2) { const float2 a = *reinterpret_cast<const float2*>(row + lane * 2); x[0] = a.x; x[1] = a.y; }
        else {
#pragma unroll
            for (int i = 0; i < C; i += 4) {
                const float4 a = *reinterpret_cast<const float4*>(row + (i >> 2) * 128 + lane * 4);
                x[i] = a.x; x[i + 1] = a.y; x[i + 2] = a.z; x[i + 3] = a.w;
            }
        }
    };
    auto row_times = [&](const float4& a, const float4& b, const float (&x)[GS_T]) {
        const float s0 = fmaf(a.y, x[1], a.x * x[0]), s1 = fmaf(a.w, x[3], a.z * x[2]);
        const float s2 = fmaf(b.y, x[5], b.x * x[4]), s3 = fmaf(b.w, x[7], b.z * x[6]);
        return (s0 + s1) + (s2 + s3);
    };
    // Sums over the lanes of N values a lane (8, 16 or 32), each exchange halving what a lane holds. A lane ends with value
    // lane / (32 / N).
    auto sums = [&](auto& p, auto count) {
        constexpr int N = decltype(count)::value;
#pragma unroll
        for (int half = N / 2, o = 16; half > 0; half >>= 1, o >>= 1) {
            const bool up = (lane & o) != 0;
#pragma unroll
            for (int i = 0; i < N / 2; ++i) {
                if (i >= half) continue;
                const float recv = __shfl_xor_sync(0xffffffffu, up ? p[i] : p[i + half], o);
                p[i] = (up ? p[i + half] : p[i]) + recv;
            }
        }
        float x = p[0];
#pragma unroll
        for (int o = 32 / N / 2; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
        return x;
    };
    // What the dot products with S read of a group sits in registers before the group's turn: it is fetched while the group
    // before is still exchanging its sums.
    float qd[GS_T][C], kd[DELTA ? GS_T : 1][C];
    auto fetch = [&](const float* st) {
#pragma unroll
        for (int t = 0; t < GS_T; ++t) {
            if constexpr (DELTA) take(st + L::K0 + t * DKP, kd[t]);
            take(st + L::Q0 + t * DKP, qd[t]);
        }
    };
    auto arrived = [&](int g) {
        const bool ok = __all_sync(0xffffffffu, mbar_wait(&full[g % STAGES], (g / STAGES) & 1));
        if (!ok) {
            if (lane == 0) atomicCAS(&g_group_walk_error, 0, (1 << 16) | (int)(blockIdx.x & 0xffff));
            s_failed = 1;
        }
        return ok;
    };
    constexpr int N = (DELTA ? 2 : 1) * NC * GS_T, EACH = 32 / N;      // sums per group: (DELTA: both dot products) x channels x tokens
    const int token = (lane / EACH) % GS_T, mine_n = (lane / EACH) / GS_T % NC;        // whose sum this lane ends with
    const bool writer = lane % EACH == 0 && (!DELTA || lane >= 16) && j0 + mine_n < cols;
    const int my_col = warp * NC + mine_n, my_j = j0 + mine_n;
    const bool my_one = ones != 0 && my_j == dv;        // the column of ones
    bool ok = true;
    if (groups > 0) {
        ok = arrived(0);
        fetch(gs_smem);
    }
    for (int g = 0; g < groups && ok; ++g) {
        const int base = row0 + g * GS_T;
        const float* st = gs_smem + (g % STAGES) * L::SIZE;
        const float* vs = s_v[g % STAGES];
        float p[N];
#pragma unroll
        for (int n = 0; n < NC; ++n)
#pragma unroll
            for (int t = 0; t < GS_T; ++t) {
                float pa = 0.f, pb = 0.f;
#pragma unroll
                for (int i = 0; i < C; ++i) {
                    if constexpr (DELTA) pa = fmaf(kd[DELTA ? t : 0][i], S[n][i], pa);
                    pb = fmaf(qd[t][i], S[n][i], pb);
                }
                if constexpr (DELTA) p[n * GS_T + t] = pa;
                p[(DELTA ? NC * GS_T : 0) + n * GS_T + t] = pb;
            }
        float ks[GS_T][C], wn[C], x[NC][GS_T];      // x: u of the group's tokens, known to every lane
#pragma unroll
        for (int t = 0; t < GS_T; ++t) take(st + L::S0 + t * DKP, ks[t]);
        take(st + L::W0, wn);
        const float4 d0 = *reinterpret_cast<const float4*>(st + L::D0 + token * GS_T), d1 = *reinterpret_cast<const float4*>(st + L::D0 + token * GS_T + 4);
        float4 a0, a1;
        float mine = 0.f;
        if constexpr (DELTA) {
            a0 = *reinterpret_cast<const float4*>(st + L::A0 + token * GS_T);
            a1 = *reinterpret_cast<const float4*>(st + L::A0 + token * GS_T + 4);
            mine = my_one ? 1.0f : vs[my_col * GS_T + token];
        } else {
#pragma unroll
            for (int n = 0; n < NC; ++n) {
                const float4 va = *reinterpret_cast<const float4*>(vs + (warp * NC + n) * GS_T), vb = *reinterpret_cast<const float4*>(vs + (warp * NC + n) * GS_T + 4);
                const bool one = ones != 0 && j0 + n == dv;
                x[n][0] = one ? 1.f : va.x; x[n][1] = one ? 1.f : va.y; x[n][2] = one ? 1.f : va.z; x[n][3] = one ? 1.f : va.w;
                x[n][4] = one ? 1.f : vb.x; x[n][5] = one ? 1.f : vb.y; x[n][6] = one ? 1.f : vb.z; x[n][7] = one ? 1.f : vb.w;
            }
        }
#pragma unroll
        for (int n = 0; n < NC; ++n)
#pragma unroll
            for (int i = 0; i < C; ++i) S[n][i] *= wn[i];
        // DELTA: the lower half of the lanes ends with (W k)^T S_0 of their channel and token, the upper half with (W q)^T S_0
        const float val = sums(p, std::integral_constant<int, N>{});
        __syncwarp();
        if (lane == 0) mbar_arrive(&empty[g % STAGES]);     // this warp has read what it needs of the group
        if (g + 1 < groups) {
            ok = arrived(g + 1);
            fetch(gs_smem + ((g + 1) % STAGES) * L::SIZE);
        }
        auto of_mine = [&](float (&y)[GS_T]) {      // x of this lane's channel
#pragma unroll
            for (int t = 0; t < GS_T; ++t) y[t] = NC == 2 && mine_n != 0 ? x[NC - 1][t] : x[0][t];
        };
        float y[GS_T];
        if constexpr (DELTA) {
            mine -= val;
#pragma unroll
            for (int n = 0; n < NC; ++n)
#pragma unroll
                for (int t = 0; t < GS_T; ++t) x[n][t] = __shfl_sync(0xffffffffu, mine, (n * GS_T + t) * EACH);
            of_mine(y);
            const float um = row_times(a0, a1, y);
#pragma unroll
            for (int n = 0; n < NC; ++n)
#pragma unroll
                for (int t = 0; t < GS_T; ++t) x[n][t] = __shfl_sync(0xffffffffu, um, (n * GS_T + t) * EACH);
        }
#pragma unroll
        for (int t = 0; t < GS_T; ++t)
#pragma unroll
            for (int n = 0; n < NC; ++n)
#pragma unroll
                for (int i = 0; i < C; ++i) S[n][i] = fmaf(ks[t][i], x[n][t], S[n][i]);
        of_mine(y);
        const float out = val + row_times(d0, d1, y);
        if (writer && base + token < row1)
            o[(size_t)(base + token) * ldo + (my_one ? (size_t)heads * dv + h : (size_t)h * dv + my_j)] = out;
    }
    pdl_launch_dependents();        // only now: blocks of the next kernel that became resident earlier would sit beside a long walk
#pragma unroll
    for (int n = 0; n < NC; ++n)
#pragma unroll
        for (int i = 0; i < C; ++i)
            if (j0 + n < cols && channel(i) < dk) head_state[(long long)(j0 + n) * dk + channel(i)] = S[n][i];
}

template <int CPL, bool DELTA>
__global__ void __launch_bounds__(128)
state_step_kernel(const float* __restrict__ q, int ldq, const float* __restrict__ k, int ldk, const float* __restrict__ v, int ldv,
                  const float* __restrict__ z, int ldz, int z_kind, const float* __restrict__ dt_bias, const float* __restrict__ rate,
                  const float* __restrict__ b, int ldb, const float* __restrict__ k_scale, float* __restrict__ state, long long state_ld,
                  int state_off, const int* __restrict__ q_start, const int* __restrict__ slots, float* __restrict__ o, int ldo, int heads,
                  int kq_heads, int dk, int dv, int ones, float q_scale, float unit_eps) {
    constexpr int NC = GS_STEP_COLS;
    pdl_launch_dependents();
    pdl_wait();      // everything this kernel reads may come from the kernel before
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, req = blockIdx.z, h = blockIdx.y;
    const int cols = dv + ones, j0 = (blockIdx.x * 4 + warp) * NC;
    const int row0 = q_start[req], row1 = q_start[req + 1];
    if (row0 >= row1 || j0 >= cols) return;     // a whole warp leaves together, and nothing below waits for the block
    float* head_state = state + (long long)slots[req] * state_ld + state_off + (long long)h * cols * dk;
    const int hq = h / (heads / kq_heads);
    const float r = z_kind == GS_STEP ? rate[h] : 0.f;
    float S[NC][CPL], bias[CPL];
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
        const int c = lane + 32 * i;
        bias[i] = (z_kind == GS_STEP && c < dk) ? dt_bias[(size_t)h * dk + c] : 0.f;
#pragma unroll
        for (int n = 0; n < NC; ++n) S[n][i] = (c < dk && j0 + n < cols) ? head_state[(long long)(j0 + n) * dk + c] : 0.f;
    }
    for (int row = row0; row < row1; ++row) {
        float kv[CPL], qv[CPL], w[CPL], val[NC];
        const float wh = z_kind == GS_HEAD ? z[(size_t)row * ldz + h] : 1.f;
        const float ks = k_scale != nullptr ? k_scale[(size_t)row * heads + h] : 1.f;
        const float zb = DELTA ? b[(size_t)row * ldb + h] : 0.f;
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
            const int c = lane + 32 * i;
            const bool in = c < dk;
            kv[i] = in ? k[(size_t)row * ldk + (size_t)hq * dk + c] : 0.f;
            qv[i] = in ? q[(size_t)row * ldq + (size_t)hq * dk + c] : 0.f;
            w[i] = !in ? 1.f : (z_kind == GS_HEAD ? wh : z[(size_t)row * ldz + (size_t)h * dk + c]);
        }
#pragma unroll
        for (int n = 0; n < NC; ++n)    // (a column of ones lies behind the others)
            val[n] = j0 + n < dv ? v[(size_t)row * ldv + (size_t)h * dv + j0 + n] : 1.f;
        float ik = ks, iq = q_scale;
        if (unit_eps >= 0.f) {
            float sk = 0.f, sq = 0.f;
#pragma unroll
            for (int i = 0; i < CPL; ++i) { sk = fmaf(kv[i], kv[i], sk); sq = fmaf(qv[i], qv[i], sq); }
            ik = ks / sqrtf(warp_sum(sk) + unit_eps);
            iq = q_scale / sqrtf(warp_sum(sq) + unit_eps);
        }
        float kq = 0.f, a[NC], out[NC];
#pragma unroll
        for (int n = 0; n < NC; ++n) a[n] = out[n] = 0.f;
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
            if (z_kind == GS_STEP && lane + 32 * i < dk) w[i] = gs_step_decay(w[i] + bias[i], r);
            kv[i] *= ik;
            qv[i] *= iq;
            kq = fmaf(kv[i], qv[i], kq);
#pragma unroll
            for (int n = 0; n < NC; ++n) {
                S[n][i] *= w[i];
                if (DELTA) a[n] = fmaf(S[n][i], kv[i], a[n]);
                out[n] = fmaf(S[n][i], qv[i], out[n]);
            }
        }
        kq = warp_sum(kq);
        const float beta = DELTA ? 1.0f / (1.0f + expf(-zb)) : 1.0f;
#pragma unroll
        for (int n = 0; n < NC; ++n) {
            const float u = DELTA ? beta * (val[n] - warp_sum(a[n])) : val[n];
            out[n] = fmaf(u, kq, warp_sum(out[n]));
#pragma unroll
            for (int i = 0; i < CPL; ++i) S[n][i] = fmaf(kv[i], u, S[n][i]);
        }
#pragma unroll
        for (int n = 0; n < NC; ++n)
            if (lane == n && j0 + n < cols)
                o[(size_t)row * ldo + (j0 + n < dv ? (size_t)h * dv + j0 + n : (size_t)heads * dv + h)] = out[n];
    }
#pragma unroll
    for (int n = 0; n < NC; ++n)
#pragma unroll
        for (int i = 0; i < CPL; ++i)
            if (lane + 32 * i < dk && j0 + n < cols) head_state[(long long)(j0 + n) * dk + lane + 32 * i] = S[n][i];
}

namespace {

template <int CPL, bool DELTA>
int launch_group(const float* q, int ldq, const float* k, int ldk, const float* v, int ldv, const float* z, int ldz, int z_kind, const float* dt_bias,
                 const float* rate, const float* b, int ldb, const float* k_scale, float* state, long long state_ld, int state_off, const int* q_start,
                 const int* slots, float* o, int ldo, float* work, int n_req, int longest, int heads, int kq_heads, int dk, int dv, int ones,
                 float q_scale, float unit_eps, cudaStream_t stream) {
    using L = GsLayout<CPL, DELTA>;
    if (longest <= GS_STEP_TOKENS) {
        NIB_CUDA(launch_pdl(state_step_kernel<CPL, DELTA>, dim3(ceil_div(dv + ones, 4 * GS_STEP_COLS), heads, n_req), dim3(128), (size_t)0, stream, q, ldq,
                            k, ldk, v, ldv, z, ldz, z_kind, dt_bias, rate, b, ldb, k_scale, state, state_ld, state_off, q_start, slots, o, ldo, heads,
                            kq_heads, dk, dv, ones, q_scale, unit_eps));
        NIB_LAUNCH_CHECK();
        return 0;
    }
    static bool configured = false;
    if (!configured) {
        NIB_CUDA(cudaFuncSetAttribute(group_walk_kernel<CPL, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::BYTES));
        configured = true;
    }
    const dim3 pgrid(ceil_div((long long)ceil_div(longest, GS_T) * heads, 4), n_req);
    NIB_CUDA(launch_pdl(group_prepare_kernel<CPL, DELTA>, pgrid, dim3(128), (size_t)0, stream, q, ldq, k, ldk, z, ldz, z_kind, dt_bias, rate, b, ldb,
                        k_scale, q_start, work, heads, kq_heads, dk, q_scale, unit_eps));
    NIB_LAUNCH_CHECK();
    const dim3 grid(ceil_div(dv + ones, L::COLS), heads, n_req);
    if (longest <= 64) {
        NIB_CUDA(launch_pdl(group_walk_kernel<CPL, DELTA>, grid, dim3(L::WARPS * 32 + 32), (size_t)L::BYTES, stream, work, v, ldv, state, state_ld, state_off,
                            q_start, slots, o, ldo, heads, dk, dv, ones));
    } else {    // plainly: as a dependent its blocks would become resident wherever room is first, several to an SM
        group_walk_kernel<CPL, DELTA><<<grid, L::WARPS * 32 + 32, L::BYTES, stream>>>(work, v, ldv, state, state_ld, state_off, q_start, slots, o, ldo, heads,
                                                                                 dk, dv, ones);
    }
    NIB_LAUNCH_CHECK();
    return 0;
}

}  // namespace

// Floats of scratch for a step of these sizes (delta: the rule with beta); 0: a short step, which is one launch.
NIB_API long long nib_grouped_state_scratch(long long tokens, int n_req, int longest, int heads, int dk, int delta) {
    if (longest <= GS_STEP_TOKENS) return 0;
    const int c = dk <= 32 ? 1 : dk <= 64 ? 2 : dk <= 128 ? 4 : 8;
    const long long size = (delta ? 3 : 2) * GS_T * 32LL * c + 32LL * c + (delta ? 2 : 1) * GS_T * GS_T;
    return (tokens / GS_T + n_req) * heads * size;
}

// The error word of the walk's bounded waits (0 = none); reading it synchronises with the device and clears it.
NIB_API int nib_grouped_state_error() {
    int v = 0, zero = 0;
    if (cudaMemcpyFromSymbol(&v, g_group_walk_error, sizeof(int)) != cudaSuccess) return -1;
    if (v != 0) cudaMemcpyToSymbol(g_group_walk_error, &zero, sizeof(int));
    return v;
}

// b [tokens, heads] (logits of beta): the delta rule; null: the plain rule. q, k: [tokens, kq_heads * dk]; z: [tokens, heads * dk] or
// [tokens, heads] (GS_HEAD); v: [tokens, heads * dv], o: [tokens, heads * dv], with ones another heads columns behind them; all floats with row strides. unit_eps >= 0:
// q and k are made unit vectors here (x / sqrt(sum x^2 + unit_eps)); queries times q_scale; k_scale [tokens, heads] or null: a factor
// on the keys. ones 1: the state has one more value channel whose value is 1. longest: the most tokens a request brings.
NIB_API int nib_grouped_state_scan(const float* q, int ldq, const float* k, int ldk, const float* v, int ldv, const float* z, int ldz, int z_kind,
                                   const float* dt_bias, const float* rate, const float* b, int ldb, const float* k_scale, float* state,
                                   long long state_ld, int state_off, const int* q_start, const int* slots, float* o, int ldo, float* scratch,
                                   int tokens, int n_req, int longest, int heads, int kq_heads, int dk, int dv, int ones, float q_scale,
                                   float unit_eps, cudaStream_t stream) {
    NIB_REQUIRE(heads > 0 && heads <= 65535 && kq_heads > 0 && heads % kq_heads == 0, "grouped_state_scan: %d heads do not share %d key heads", heads, kq_heads);
    NIB_REQUIRE(dk > 0 && dk <= 256 && dv > 0 && (ones == 0 || ones == 1), "grouped_state_scan: key size %d is outside 1..256", dk);
    NIB_REQUIRE(z_kind >= GS_STEP && z_kind <= GS_HEAD && (z_kind != GS_STEP || (rate != nullptr && dt_bias != nullptr)) && (scratch != nullptr || longest <= GS_STEP_TOKENS)
                && ((uintptr_t)scratch & 15) == 0, "grouped_state_scan: bad arguments");
    if (n_req <= 0 || tokens <= 0) return 0;
    NIB_REQUIRE(longest > 0 && n_req <= 65535, "grouped_state_scan: bad batch");
#define NIB_GS(CPL, DELTA) launch_group<CPL, DELTA>(q, ldq, k, ldk, v, ldv, z, ldz, z_kind, dt_bias, rate, b, ldb, k_scale, state, state_ld, state_off, \
                                                    q_start, slots, o, ldo, scratch, n_req, longest, heads, kq_heads, dk, dv, ones, q_scale, unit_eps, stream)
    if (b != nullptr) return dk <= 32 ? NIB_GS(1, true) : dk <= 64 ? NIB_GS(2, true) : dk <= 128 ? NIB_GS(4, true) : NIB_GS(8, true);
    return dk <= 32 ? NIB_GS(1, false) : dk <= 64 ? NIB_GS(2, false) : dk <= 128 ? NIB_GS(4, false) : NIB_GS(8, false);
#undef NIB_GS
}

// ---------------------------------------------------------------------------------- gates of a stabilized matrix memory
// Per (token, head): the log input gate i = cap * tanh((zi + bi) / cap), the log forget gate f = log sigmoid(cap * tanh((zf +
// bf) / cap)), and the running maximum m_t = max(f + m_(t-1), i), which starts at the state's number (zero at a request's
// start) and is kept there. Out: decay = exp(f + m_(t-1) - m_t), write = exp(i - m_t), floor = exp(-m_t). A block per
// (request, head), a thread per token: the maxima are a scan over the maps m -> max(m + F, A), composed in warps, then across the
// block's warps. Whatever m_t was rounded to, decay and write are formed from the m's as they are, the exponent of the decay
// without rounding its sum (the part that an addition loses is added back), so that along a sequence the weight of an
// old token against a new one is the sum of the f between them.
__global__ void __launch_bounds__(1024)
memory_gates_kernel(const float* __restrict__ zi, int ldi, const float* __restrict__ zf, int ldf, const float* __restrict__ bi,
                    const float* __restrict__ bf, float cap, float* __restrict__ state, long long state_ld, int state_off,
                    const int* __restrict__ q_start, const int* __restrict__ slots, float* __restrict__ decay, float* __restrict__ write,
                    float* __restrict__ floor_out, int heads) {
    __shared__ float s_f[32], s_a[32], s_m[32];
    pdl_launch_dependents();
    pdl_wait();      // everything this kernel reads may come from the kernel before
    const int h = blockIdx.x, req = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int row0 = q_start[req], row1 = q_start[req + 1];
    if (row0 >= row1) return;
    float* st = state + (long long)slots[req] * state_ld + state_off + h;
    float m_in = *st;
    for (int base = row0; base < row1; base += blockDim.x) {
        const int t = base + threadIdx.x;
        const bool live = t < row1;
        float i = 0.f, f = 0.f;
        if (live) {
            i = cap * tanhf((zi[(size_t)t * ldi + h] + bi[h]) / cap);
            const float x = cap * tanhf((zf[(size_t)t * ldf + h] + bf[h]) / cap);
            f = x >= 0.f ? -log1pf(expf(-x)) : x - log1pf(expf(x));
        }
        // the maps of this warp's tokens, composed: m -> max(m + F, A)
        float F = f, A = live ? i : -INFINITY;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pF = __shfl_up_sync(0xffffffffu, F, o), pA = __shfl_up_sync(0xffffffffu, A, o);
            if (lane >= o) { A = fmaxf(pA + F, A); F += pF; }
        }
        if (lane == 31) { s_f[warp] = F; s_a[warp] = A; }
        __syncthreads();
        float m0 = m_in;
        for (int w = 0; w < warp; ++w) m0 = fmaxf(m0 + s_f[w], s_a[w]);
        const float m = fmaxf(m0 + F, A);
        float before = __shfl_up_sync(0xffffffffu, m, 1);
        if (lane == 31) s_m[warp] = m;
        __syncthreads();
        if (lane == 0) before = warp == 0 ? m_in : s_m[warp - 1];
        if (live) {
            const size_t at = (size_t)t * heads + h;
            // before + f as a rounded sum and what the rounding lost
            const float sum = before + f, back = sum - before, lost = (before - (sum - back)) + (f - back);
            decay[at] = gs_decay_exp((sum - m) + lost);
            write[at] = expf(i - m);
            floor_out[at] = expf(-m);
            if (t == row1 - 1) *st = m;
        }
        m_in = s_m[warps - 1];      // (a block that goes on is full: its last thread holds a token)
        __syncthreads();
    }
}

NIB_API int nib_memory_gates(const float* zi, int ldi, const float* zf, int ldf, const float* bi, const float* bf, float cap, float* state,
                             long long state_ld, int state_off, const int* q_start, const int* slots, float* decay, float* write,
                             float* floor_out, int n_req, int longest, int heads, cudaStream_t stream) {
    NIB_REQUIRE(n_req >= 0 && n_req <= 65535 && heads > 0 && cap > 0.f && bi != nullptr && bf != nullptr, "memory_gates: bad sizes");
    if (n_req == 0 || longest <= 0) return 0;
    const int threads = longest >= 1024 ? 1024 : ((longest + 31) / 32) * 32;
    NIB_CUDA(launch_pdl(memory_gates_kernel, dim3(heads, n_req), dim3(threads), (size_t)0, stream, zi, ldi, zf, ldf, bi, bf, cap, state, state_ld,
                        state_off, q_start, slots, decay, write, floor_out, heads));
    NIB_LAUNCH_CHECK();
    return 0;
}
