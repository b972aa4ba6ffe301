// The gated delta rule over a flat batch of requests: per head a matrix state S [key channel x value channel] that decays
// by rows, gives up the part of the token's value that it already answers to the token's key, and takes the rest:
//
//     S <- diag(w_t) S,   u_t = beta_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   o_t = S^T q_t      (all 32-bit)
//
// A request brings a prompt's portion or one decoded token; its state is a row of floats in a slot of a state tensor (row
// stride `state_ld`, from column `state_off`, laid out [head, value channel, key channel]). Which request owns which rows
// and which slot is read from device arrays, so a captured graph can replay the launches for other requests.
//
// A request's tokens are taken DS_T at a time. Within such a group everything that does not involve S can be known before
// S is: with W_t the product of the group's decays up to and including token t, and with W_(s,t] the product of those
// after s up to t,
//
//     u_t = beta_t (v_t - (W_t k_t)^T S_0 - sum_(s<t) c_ts u_s),     c_ts = sum_ch k_t k_s W_(s,t],
//     o_t = (W_t q_t)^T S_0 + sum_(s<=t) d_ts u_s,                   d_ts = sum_ch q_t k_s W_(s,t],
//     S_n = W_n S_0 + sum_s (W_(s,n] k_s) u_s^T,
//
// so u = A (v - (W k)^T S_0) with A = (I + diag(beta) C)^(-1) diag(beta), a lower triangular matrix per (group, head) that all
// value channels share. Only products of decays appear (no quotients), so strong decays underflow to zero harmlessly.
//  * delta_prepare: a warp per (group, head): unit keys and queries, decays, beta, the vectors W_t k_t, W_t q_t, W_(s,n] k_s,
//    W_n, and the matrices A and D; parallel over the whole step.
//  * delta_walk: a block owns 16 value channels of a head of a request, eight lanes share a channel (its key channels in
//    registers) and walk the groups in order: two dot products per token with S_0, one butterfly for the eight tokens' sums
//    together, two 8 x 8 products with the matrices, one update of S per group.
// Groups start at the step's first token of a request: a result depends on how the request was cut by rounding only.
#include "common.cuh"

constexpr int DS_T = 8;             // tokens per group: as many as lanes share a value channel
constexpr int DS_COLS = 16;
constexpr int DS_LANES = 8;
constexpr int DS_THREADS = DS_COLS * DS_LANES;

// Scratch, all by token row (row strides heads * dk resp. heads * DS_T): kd = W_t k_t, qd = W_t q_t, ks = W_(t,n] k_t,
// wn = W_n (in the row of a group's first token), a = rows of A, d = rows of D. a and d come first: their rows of eight
// floats then start on 16-byte boundaries whatever dk is.
struct DeltaWork { float *kd, *qd, *ks, *wn, *a, *d; };

static __host__ __device__ inline DeltaWork delta_work(float* base, long long tokens, int heads, int dk) {
    const long long plane = tokens * heads * dk, small = tokens * heads * DS_T;
    float* vectors = base + 2 * small;
    return DeltaWork{vectors, vectors + plane, vectors + 2 * plane, vectors + 3 * plane, base, base + small};
}

__device__ __forceinline__ float ds_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }

// z: with a_log, the logits of the step sizes (decay = exp(-exp(a_log[h]) * softplus(z + dt_bias)), rounded to 32 bits once
// from 64-bit exponentials: a decay is raised to hundreds of powers along a sequence); without, the decays themselves.
template <int CPL>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const float* __restrict__ q, int ldq, const float* __restrict__ k, int ldk, const float* __restrict__ z, int ldz,
                     const float* __restrict__ dt_bias, const float* __restrict__ a_log, const float* __restrict__ b, int ldb,
                     const int* __restrict__ q_start, DeltaWork work, int heads, int kq_heads, int dk, float q_scale, float unit_eps) {
    pdl_launch_dependents();
    pdl_wait();      // everything this kernel reads may come from the kernel before
    __shared__ float s_m[4][DS_T * DS_T];       // per warp: D on and below the diagonal, C mirrored above it
    __shared__ float s_beta[4][DS_T];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, req = blockIdx.y;
    const int wid = blockIdx.x * 4 + warp;
    const int group = wid / heads, h = wid - group * heads;
    const int first = q_start[req], len = q_start[req + 1] - first;
    if (group * DS_T >= len) return;            // a whole warp leaves together, and nothing below waits for the block
    const int row0 = first + group * DS_T, nt = min(DS_T, len - group * DS_T);
    const int hq = h / (heads / kq_heads);
    const double rate = a_log != nullptr ? exp((double)a_log[h]) : 0.0;
    float run[DS_T][CPL];       // k_s times the decays after s so far
    float pre[CPL];             // the product of the decays so far
    float acc[DS_T * DS_T];
#pragma unroll
    for (int i = 0; i < DS_T * DS_T; ++i) acc[i] = 0.f;
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
        pre[i] = 1.f;
#pragma unroll
        for (int s = 0; s < DS_T; ++s) run[s][i] = 0.f;
    }
#pragma unroll
    for (int t = 0; t < DS_T; ++t) {
        if (t >= nt) continue;
        const size_t row = (size_t)(row0 + t);
        float kv[CPL], qv[CPL], sk = 0.f, sq = 0.f;
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
            const int c = lane + 32 * i;
            kv[i] = c < dk ? k[row * ldk + (size_t)hq * dk + c] : 0.f;
            qv[i] = c < dk ? q[row * ldq + (size_t)hq * dk + c] : 0.f;
            sk = fmaf(kv[i], kv[i], sk);
            sq = fmaf(qv[i], qv[i], sq);
        }
        const float ik = 1.0f / sqrtf(warp_sum(sk) + unit_eps), iq = q_scale / sqrtf(warp_sum(sq) + unit_eps);
        if (lane == 0) s_beta[warp][t] = ds_sigmoid(b[row * ldb + h]);
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
            const int c = lane + 32 * i;
            float w = 1.f;
            if (c < dk) {
                w = z[row * ldz + (size_t)h * dk + c];
                if (a_log != nullptr) {
                    const double x = (double)(w + dt_bias[(size_t)h * dk + c]);
                    const double step = x > 0.0 ? x + log1p(exp(-x)) : log1p(exp(x));
                    w = (float)exp(-rate * step);
                }
            }
            kv[i] *= ik;
            qv[i] *= iq;
            pre[i] *= w;
#pragma unroll
            for (int s = 0; s < DS_T; ++s) {
                if (s < t) {
                    run[s][i] *= w;
                    acc[t * DS_T + s] = fmaf(qv[i], run[s][i], acc[t * DS_T + s]);
                    acc[s * DS_T + t] = fmaf(kv[i], run[s][i], acc[s * DS_T + t]);
                }
            }
            run[t][i] = kv[i];
            acc[t * DS_T + t] = fmaf(qv[i], kv[i], acc[t * DS_T + t]);
            if (c < dk) {
                const size_t at = row * heads * dk + (size_t)h * dk + c;
                work.kd[at] = kv[i] * pre[i];
                work.qd[at] = qv[i] * pre[i];
            }
        }
    }
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
        const int c = lane + 32 * i;
        if (c >= dk) continue;
#pragma unroll
        for (int s = 0; s < DS_T; ++s)
            if (s < nt) work.ks[(size_t)(row0 + s) * heads * dk + (size_t)h * dk + c] = run[s][i];
        work.wn[(size_t)row0 * heads * dk + (size_t)h * dk + c] = pre[i];
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
    if (lane < DS_T) {
        // column `lane` of A by forward substitution: x_t = beta_t ([t == lane] - sum_(s<t) c_ts x_s); row `lane` of D
        float x[DS_T];
#pragma unroll
        for (int t = 0; t < DS_T; ++t) {
            float sum = t == lane ? 1.f : 0.f;
#pragma unroll
            for (int s = 0; s < DS_T; ++s)
                if (s < t) sum = fmaf(-m[s * DS_T + t], x[s], sum);
            x[t] = t < nt ? s_beta[warp][t] * sum : 0.f;
            if (t < nt) work.a[((size_t)(row0 + t) * heads + h) * DS_T + lane] = x[t];
        }
        if (lane < nt) {
            float* d = work.d + ((size_t)(row0 + lane) * heads + h) * DS_T;
#pragma unroll
            for (int s = 0; s < DS_T; ++s) d[s] = s <= lane ? m[lane * DS_T + s] : 0.f;
        }
    }
}

__device__ __forceinline__ void ds_cp_async(void* smem, const void* gmem, bool valid, bool wide) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    if (wide) {
        const int n = valid ? 16 : 0;       // 0 source bytes: the destination is zero-filled
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(n));
    } else {
        const int n = valid ? 4 : 0;
        asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"(s), "l"(gmem), "r"(n));
    }
}

// One staged group: kd, qd, ks (DS_T rows of DKP floats each), wn, the block's value columns, A and D.
template <int C> struct DsLayout {
    static constexpr int DKP = DS_LANES * C;
    static constexpr int Q0 = DS_T * DKP, S0 = 2 * DS_T * DKP, W0 = 3 * DS_T * DKP, V0 = W0 + DKP, A0 = V0 + DS_T * DS_COLS,
                         D0 = A0 + DS_T * DS_T, STAGE = D0 + DS_T * DS_T;
    static constexpr int STAGES = C >= 32 ? 3 : 4;
    static constexpr int BYTES = STAGES * STAGE * 4;
};

template <int C>
__global__ void __launch_bounds__(DS_THREADS)
delta_walk_kernel(const DeltaWork work, const float* __restrict__ v, int ldv, float* __restrict__ state, long long state_ld, int state_off,
                  const int* __restrict__ q_start, const int* __restrict__ slots, float* __restrict__ o, int ldo, int heads, int dk, int dv,
                  int wide) {
    using L = DsLayout<C>;
    constexpr int DKP = L::DKP, STAGES = L::STAGES;
    extern __shared__ __align__(16) float ds_smem[];
    const int req = blockIdx.z, h = blockIdx.y;
    const int lane = threadIdx.x & (DS_LANES - 1), col = threadIdx.x / DS_LANES, j = blockIdx.x * DS_COLS + col;
    const bool live = j < dv;
    const int row0 = q_start[req], row1 = q_start[req + 1];
    pdl_wait();      // everything below may come from the kernels before
    float* srow = state + (long long)slots[req] * state_ld + state_off + ((long long)h * dv + (live ? j : 0)) * dk;
    // lane l owns the key channels (8 i + l) * 4 .. + 3: the eight lanes read 128 consecutive bytes of a vector per load
    float S[C];
#pragma unroll
    for (int i = 0; i < C; ++i) {
        const int c = ((i >> 2) * DS_LANES + lane) * 4 + (i & 3);
        S[i] = (live && c < dk) ? srow[c] : 0.f;
    }
    auto stage = [&](int buf, int base) {
        float* st = ds_smem + buf * L::STAGE;
        const int nt = min(DS_T, row1 - base);
        const int step = wide ? 4 : 1, per = DKP / step;
        for (int e = threadIdx.x; e < DS_T * per; e += DS_THREADS) {
            const int tt = e / per, c = (e - tt * per) * step;
            const bool ok = tt < nt && c < dk;
            const size_t at = (size_t)(base + (ok ? tt : 0)) * heads * dk + (size_t)h * dk + (ok ? c : 0);
            ds_cp_async(st + tt * DKP + c, work.kd + at, ok, wide);
            ds_cp_async(st + L::Q0 + tt * DKP + c, work.qd + at, ok, wide);
            ds_cp_async(st + L::S0 + tt * DKP + c, work.ks + at, ok, wide);
            if (tt == 0) ds_cp_async(st + L::W0 + c, work.wn + at, ok, wide);
        }
        for (int e = threadIdx.x; e < DS_T * DS_COLS; e += DS_THREADS) {
            const int tt = e / DS_COLS, cc = e % DS_COLS, jj = blockIdx.x * DS_COLS + cc;
            const bool ok = tt < nt && jj < dv;
            ds_cp_async(st + L::V0 + e, v + (size_t)(base + (ok ? tt : 0)) * ldv + (size_t)h * dv + (ok ? jj : 0), ok, false);
        }
        if (threadIdx.x < 2 * DS_T * DS_T / 4) {        // rows of A, then rows of D, four floats a thread
            const int e = threadIdx.x & (DS_T * DS_T / 4 - 1), tt = e / 2, c = (e & 1) * 4;
            const bool is_d = threadIdx.x >= DS_T * DS_T / 4, ok = tt < nt;
            ds_cp_async(st + (is_d ? L::D0 : L::A0) + tt * DS_T + c,
                        (is_d ? work.d : work.a) + ((size_t)(base + (ok ? tt : 0)) * heads + h) * DS_T + c, ok, true);
        }
    };
    for (int st = 0; st < STAGES - 1; ++st) {
        if (row0 + st * DS_T < row1) stage(st, row0 + st * DS_T);
        asm volatile("cp.async.commit_group;\n" ::);
    }
    const bool up4 = (lane & 4) != 0, up2 = (lane & 2) != 0, up1 = (lane & 1) != 0;
    // eight lanes' shares of eight sums, in three exchanges: lane l ends with sum l
    auto gather = [&](const float (&p)[DS_T]) {
        float h4[4], h2[2];
#pragma unroll
        for (int t = 0; t < 4; ++t) h4[t] = (up4 ? p[t + 4] : p[t]) + __shfl_xor_sync(0xffffffffu, up4 ? p[t] : p[t + 4], 4);
#pragma unroll
        for (int t = 0; t < 2; ++t) h2[t] = (up2 ? h4[t + 2] : h4[t]) + __shfl_xor_sync(0xffffffffu, up2 ? h4[t] : h4[t + 2], 2);
        return (up1 ? h2[1] : h2[0]) + __shfl_xor_sync(0xffffffffu, up1 ? h2[0] : h2[1], 1);
    };
    auto row_times = [&](const float* m, const float (&x)[DS_T]) {     // row `lane` of an 8 x 8 matrix times x
        const float4 a = *reinterpret_cast<const float4*>(m + lane * DS_T), b = *reinterpret_cast<const float4*>(m + lane * DS_T + 4);
        const float s0 = fmaf(a.y, x[1], a.x * x[0]), s1 = fmaf(a.w, x[3], a.z * x[2]);
        const float s2 = fmaf(b.y, x[5], b.x * x[4]), s3 = fmaf(b.w, x[7], b.z * x[6]);
        return (s0 + s1) + (s2 + s3);
    };
    int buf = 0;
    for (int base = row0; base < row1; base += DS_T, buf = (buf + 1 == STAGES ? 0 : buf + 1)) {
        const int nt = min(DS_T, row1 - base), ahead = base + (STAGES - 1) * DS_T;
        if (ahead < row1) stage(buf == 0 ? STAGES - 1 : buf - 1, ahead);
        asm volatile("cp.async.commit_group;\n" ::);
        asm volatile("cp.async.wait_group %0;\n" ::"n"(STAGES - 1));
        __syncthreads();
        const float* st = ds_smem + buf * L::STAGE;
        float p[DS_T], r[DS_T];
#pragma unroll
        for (int t = 0; t < DS_T; ++t) {
            float pa = 0.f, pb = 0.f, ra = 0.f, rb = 0.f;
#pragma unroll
            for (int i4 = 0; i4 < C / 4; ++i4) {
                const int c4 = (i4 * DS_LANES + lane) * 4;
                const float4 kd = *reinterpret_cast<const float4*>(st + t * DKP + c4), qd = *reinterpret_cast<const float4*>(st + L::Q0 + t * DKP + c4);
                pa = fmaf(kd.x, S[4 * i4], pa); pb = fmaf(kd.y, S[4 * i4 + 1], pb); pa = fmaf(kd.z, S[4 * i4 + 2], pa); pb = fmaf(kd.w, S[4 * i4 + 3], pb);
                ra = fmaf(qd.x, S[4 * i4], ra); rb = fmaf(qd.y, S[4 * i4 + 1], rb); ra = fmaf(qd.z, S[4 * i4 + 2], ra); rb = fmaf(qd.w, S[4 * i4 + 3], rb);
            }
            p[t] = pa + pb;
            r[t] = ra + rb;
        }
        const float mine = st[L::V0 + lane * DS_COLS + col] - gather(p);       // token `lane`: v - (W k)^T S_0
        const float read = gather(r);
        float x[DS_T];
#pragma unroll
        for (int t = 0; t < DS_T; ++t) x[t] = __shfl_sync(0xffffffffu, mine, t, DS_LANES);
        const float um = row_times(st + L::A0, x);
#pragma unroll
        for (int t = 0; t < DS_T; ++t) x[t] = __shfl_sync(0xffffffffu, um, t, DS_LANES);
        const float om = read + row_times(st + L::D0, x);
        if (lane < nt && live) o[(size_t)(base + lane) * ldo + (size_t)h * dv + j] = om;
#pragma unroll
        for (int i4 = 0; i4 < C / 4; ++i4) {
            const int c4 = (i4 * DS_LANES + lane) * 4;
            const float4 wn = *reinterpret_cast<const float4*>(st + L::W0 + c4);
            float a = S[4 * i4] * wn.x, b = S[4 * i4 + 1] * wn.y, c = S[4 * i4 + 2] * wn.z, d = S[4 * i4 + 3] * wn.w;
#pragma unroll
            for (int t = 0; t < DS_T; ++t) {
                const float4 ks = *reinterpret_cast<const float4*>(st + L::S0 + t * DKP + c4);
                a = fmaf(ks.x, x[t], a); b = fmaf(ks.y, x[t], b); c = fmaf(ks.z, x[t], c); d = fmaf(ks.w, x[t], d);
            }
            S[4 * i4] = a; S[4 * i4 + 1] = b; S[4 * i4 + 2] = c; S[4 * i4 + 3] = d;
        }
        __syncthreads();        // the group has been walked: its buffer may be filled again
    }
    pdl_launch_dependents();        // only now: blocks of the next kernel that became resident earlier would sit beside a long walk
    if (live) {
#pragma unroll
        for (int i = 0; i < C; ++i) {
            const int c = ((i >> 2) * DS_LANES + lane) * 4 + (i & 3);
            if (c < dk) srow[c] = S[i];
        }
    }
}

// Floats of scratch for a step of these sizes.
NIB_API long long nib_delta_state_scratch(long long tokens, int heads, int dk) { return tokens * heads * (4LL * dk + 2 * DS_T); }

// q, k: [tokens, kq_heads * dk]; z: [tokens, heads * dk]; b: [tokens, heads] (logits of beta); v, o: [tokens, heads * dv]; all
// floats with row strides. Unit keys and queries are made here (x / sqrt(sum x^2 + unit_eps)), queries times q_scale.
// longest: the most tokens a request brings.
NIB_API int nib_delta_state_scan(const float* q, int ldq, const float* k, int ldk, const float* v, int ldv, const float* z, int ldz,
                                 const float* dt_bias, const float* a_log, const float* b, int ldb, float* state, long long state_ld,
                                 int state_off, const int* q_start, const int* slots, float* o, int ldo, float* scratch, int tokens, int n_req,
                                 int longest, int heads, int kq_heads, int dk, int dv, float q_scale, float unit_eps, cudaStream_t stream) {
    NIB_REQUIRE(heads > 0 && kq_heads > 0 && heads % kq_heads == 0, "delta_state_scan: %d heads do not share %d key heads", heads, kq_heads);
    NIB_REQUIRE(dk > 0 && dk <= 256 && dv > 0, "delta_state_scan: key size %d is outside 1..256", dk);
    NIB_REQUIRE((a_log == nullptr) == (dt_bias == nullptr) && scratch != nullptr && ((uintptr_t)scratch & 15) == 0, "delta_state_scan: bad arguments");
    if (n_req <= 0 || tokens <= 0) return 0;
    NIB_REQUIRE(longest > 0 && n_req <= 65535, "delta_state_scan: bad batch");
    const DeltaWork work = delta_work(scratch, tokens, heads, dk);
    const dim3 pgrid(ceil_div((long long)ceil_div(longest, DS_T) * heads, 4), n_req);
#define NIB_DSP(CPL) NIB_CUDA(launch_pdl(delta_prepare_kernel<CPL>, pgrid, dim3(128), (size_t)0, stream, q, ldq, k, ldk, z, ldz, dt_bias, a_log, b, ldb, q_start, work, heads, kq_heads, dk, q_scale, unit_eps))
    if (dk <= 32) NIB_DSP(1); else if (dk <= 64) NIB_DSP(2); else if (dk <= 128) NIB_DSP(4); else NIB_DSP(8);
#undef NIB_DSP
    NIB_LAUNCH_CHECK();
    const dim3 grid(ceil_div(dv, DS_COLS), heads, n_req);
    const int wide = dk % 4 == 0 ? 1 : 0;       // rows of the vectors that start on 16-byte boundaries
#define NIB_DSW(C)                                                                                                                  \
    do {                                                                                                                            \
        static bool configured = false;                                                                                             \
        if (!configured) {                                                                                                          \
            NIB_CUDA(cudaFuncSetAttribute(delta_walk_kernel<C>, cudaFuncAttributeMaxDynamicSharedMemorySize, DsLayout<C>::BYTES));  \
            configured = true;                                                                                                      \
        }                                                                                                                           \
        if (longest <= 64) {                                                                                                        \
            NIB_CUDA(launch_pdl(delta_walk_kernel<C>, grid, dim3(DS_THREADS), (size_t)DsLayout<C>::BYTES, stream, work, v, ldv,      \
                                state, state_ld, state_off, q_start, slots, o, ldo, heads, dk, dv, wide));                          \
        } else {    /* plainly: as a dependent its blocks would become resident wherever room is first, several to an SM */         \
            delta_walk_kernel<C><<<grid, DS_THREADS, DsLayout<C>::BYTES, stream>>>(work, v, ldv, state, state_ld, state_off,        \
                                                                                   q_start, slots, o, ldo, heads, dk, dv, wide);    \
        }                                                                                                                           \
    } while (0)
    if (dk <= 32) NIB_DSW(4); else if (dk <= 64) NIB_DSW(8); else if (dk <= 128) NIB_DSW(16); else NIB_DSW(32);
#undef NIB_DSW
    NIB_LAUNCH_CHECK();
    return 0;
}
