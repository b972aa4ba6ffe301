// Matrix states with ONE decay per head and token, S_t = d_t S_(t-1) + f_t k_t v_t^T, o_t = S_t^T q_t (S: key channel x value
// channel, 32-bit): the state-space mixer (d = exp(-exp(a_log) dt), f = dt, dt = softplus(raw + bias) per token) and linear attention
// with a fixed decay per head (f = 1). q, k and v may pass silu on the way in; q and k may be shared by groups of heads. State layout
// per slot: [head, value channel, key channel]. Which request owns which rows and which slot is read from device arrays, as in
// linear_state.cu.
//
// Short steps (decode_step): token by token, the state in registers, a group of lanes per four value channels.
//
// Prompts, in chunks of CH tokens from a request's first token of the step. With c_t the sum of the logarithms of the decays of
// a chunk's tokens up to t,
//     o_t = e^(c_t) S_in^T q_t + sum_(s<=t) (q_t . k_s) e^(c_t - c_s) f_s v_s,      S_out = e^(c_end) S_in + sum_s e^(c_end - c_s) f_s k_s v_s^T
// so that everything but the chain of the S_in is products of matrices:
//   chunk_state:   what a chunk adds to a zero state, and its e^(c_end); all chunks side by side
//   chunk_chain:   the entry state of every chunk, one after the other (element by element), the last state into the slot
//   chunk_output:  the outputs; all chunks side by side
// Only differences c_t - c_s <= 0 are exponentiated, never quotients of products, so a decay of zero is a zero; the sums are formed in
// 64-bit and kept as two floats, so a strong decay early in a chunk does not cost the later differences their digits.
// The products run on the tensor cores (mma.sync m16n8k16, bfloat16 operands, 32-bit sums). q, k and v are outputs of
// projections and convolutions and enter as bfloat16 (they may be stored so, T, or as floats); what is 32-bit by the design (states,
// decays, step sizes, and everything they multiply) is split into a bfloat16 and a bfloat16 of the remainder, two products each: 16
// bits and more of it take part. A block takes units, 64 value channels of a head each: two that share q and k where such pairs
// exist, else one; tiles come by cp.async where rows are aligned. What passes
// between the three kernels lies in the order of the products' fragments: a lane's eight numbers of a 16 x 16 piece of a state (value
// channels g and g + 8, key channels 2t, 2t + 1, 2t + 8, 2t + 9 of it, g = lane / 4, t = lane % 4) are 32 consecutive bytes, which
// chunk_state holds in its accumulators and chunk_output multiplies with as they come from memory.
#include "attention_common.cuh"

namespace {

constexpr int CH = 64;                  // tokens of a chunk
constexpr int DS_THREADS = 128;
constexpr float NO_DECAY_LEFT = -1e30f; // log2 of a decay of zero

struct DsIn {
    const void *q, *k, *v;              // rows of ldq, ldk, ldv elements of type T
    const float *raw, *bias, *a_log;    // step sizes: raw [tokens] rows of ld_raw floats (null: fixed decays), bias and a_log [heads]
    const float *decay, *log2_decay;    // fixed decays and their logarithms [heads]
    const int *q_start, *slots;
    int ldq, ldk, ldv, ld_raw, heads, kq_heads, dk, dv, silu, vec;
    template <typename T> __device__ __forceinline__ const T* q_at(size_t row, int head) const { return (const T*)q + row * ldq + (size_t)head * dk; }
    template <typename T> __device__ __forceinline__ const T* k_at(size_t row, int head) const { return (const T*)k + row * ldk + (size_t)head * dk; }
    template <typename T> __device__ __forceinline__ const T* v_at(size_t row, int head) const { return (const T*)v + row * ldv + (size_t)head * dv; }
};

__device__ __forceinline__ float ds_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus(float x) { return x > 0.f ? x + log1pf(expf(-x)) : log1pf(expf(x)); }

// elements c .. c + 3 of a row of `width` elements as floats, zeros beyond its end; vec: the width is a multiple of four and the
// row starts on a boundary of four elements
__device__ __forceinline__ float4 row4(const float* p, int c, int width, bool vec) {
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (vec) {
        if (c < width) x = *reinterpret_cast<const float4*>(p + c);
    } else {
        if (c < width) x.x = p[c];
        if (c + 1 < width) x.y = p[c + 1];
        if (c + 2 < width) x.z = p[c + 2];
        if (c + 3 < width) x.w = p[c + 3];
    }
    return x;
}
__device__ __forceinline__ float4 row4(const __nv_bfloat16* p, int c, int width, bool vec) {
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (vec) {
        if (c < width) {
            const uint2 raw = *reinterpret_cast<const uint2*>(p + c);
            const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
            x = make_float4(a.x, a.y, b.x, b.y);
        }
    } else {
        if (c < width) x.x = __bfloat162float(p[c]);
        if (c + 1 < width) x.y = __bfloat162float(p[c + 1]);
        if (c + 2 < width) x.z = __bfloat162float(p[c + 2]);
        if (c + 3 < width) x.w = __bfloat162float(p[c + 3]);
    }
    return x;
}
// with the fast exponential and division (2 ulp), for results that are rounded to bfloat16
__device__ __forceinline__ float silu_fast(float x) { return __fdividef(x, 1.0f + __expf(-x)); }
__device__ __forceinline__ void silu4(float4& x) { x = make_float4(silu_fast(x.x), silu_fast(x.y), silu_fast(x.z), silu_fast(x.w)); }

// ---------------------------------------------------------------------------------- short steps
// grid: (parts of the value channels, heads, requests). LANES lanes share R value channels; lane l holds the key channels
// (l + LANES i) * 4 .. + 3.
constexpr int R = 4;

template <typename T, int LANES, int NV>
__global__ void __launch_bounds__(DS_THREADS)
decay_step_kernel(const DsIn in, float* __restrict__ state, long long state_ld, int state_off, float* __restrict__ o, int ldo) {
    pdl_launch_dependents();
    const int req = blockIdx.z, h = blockIdx.y, hq = h / (in.heads / in.kq_heads);
    const int lane = threadIdx.x % LANES, j0 = (blockIdx.x * (DS_THREADS / LANES) + threadIdx.x / LANES) * R;
    const int dk = in.dk, dv = in.dv;
    const bool fixed = in.raw == nullptr;
    const float bias = fixed ? 0.f : in.bias[h], rate = fixed ? 0.f : expf(in.a_log[h]);      // weights
    const float d_fixed = fixed ? in.decay[h] : 0.f;
    pdl_wait();         // everything else this kernel reads may come from the kernel before
    const int row0 = in.q_start[req], row1 = in.q_start[req + 1];
    if (row0 >= row1) return;
    float* base = state + (long long)in.slots[req] * state_ld + state_off + ((long long)h * dv + j0) * dk;
    float S[R][NV][4];
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = (lane + LANES * i) * 4;
            const float* p = base + (long long)r * dk + c;
            S[r][i][0] = S[r][i][1] = S[r][i][2] = S[r][i][3] = 0.f;
            if (j0 + r >= dv) continue;
            if (in.vec) {
                if (c < dk) { const float4 x = *reinterpret_cast<const float4*>(p); S[r][i][0] = x.x; S[r][i][1] = x.y; S[r][i][2] = x.z; S[r][i][3] = x.w; }
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) if (c + e < dk) S[r][i][e] = p[e];
            }
        }
    for (int t = row0; t < row1; ++t) {
        float qv[NV][4], kv[NV][4], vv[R];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = (lane + LANES * i) * 4;
            const float4 a = row4(in.q_at<T>(t, hq), c, dk, in.vec != 0), b = row4(in.k_at<T>(t, hq), c, dk, in.vec != 0);
            qv[i][0] = a.x; qv[i][1] = a.y; qv[i][2] = a.z; qv[i][3] = a.w;
            kv[i][0] = b.x; kv[i][1] = b.y; kv[i][2] = b.z; kv[i][3] = b.w;
        }
#pragma unroll
        for (int r = 0; r < R; ++r) vv[r] = j0 + r < dv ? Elem<T>::load(in.v_at<T>(t, h) + j0 + r) : 0.f;
        float d = d_fixed, f = 1.0f;
        if (!fixed) {
            f = softplus(in.raw[(size_t)t * in.ld_raw + h] + bias);
            d = 1.0f + expm1f(-rate * f);       // (near one off by its own rounding alone)
        }
        if (in.silu) {
#pragma unroll
            for (int i = 0; i < NV; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) { qv[i][e] = ds_silu(qv[i][e]); kv[i][e] = ds_silu(kv[i][e]); }
#pragma unroll
            for (int r = 0; r < R; ++r) vv[r] = ds_silu(vv[r]);
        }
        float acc[R];
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const float u = vv[r] * f;
            float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i = 0; i < NV; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    S[r][i][e] = fmaf(d, S[r][i][e], kv[i][e] * u);
                    a[e] = fmaf(qv[i][e], S[r][i][e], a[e]);
                }
            acc[r] = (a[0] + a[1]) + (a[2] + a[3]);
        }
#pragma unroll
        for (int m = LANES / 2; m > 0; m >>= 1)
#pragma unroll
            for (int r = 0; r < R; ++r) acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], m);
        float mine = acc[0];
#pragma unroll
        for (int r = 1; r < R; ++r) if (lane == r) mine = acc[r];
        if (lane < R && j0 + lane < dv) o[(size_t)t * ldo + (size_t)h * dv + j0 + lane] = mine;
    }
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = (lane + LANES * i) * 4;
            float* p = base + (long long)r * dk + c;
            if (j0 + r >= dv) continue;
            if (in.vec) {
                if (c < dk) *reinterpret_cast<float4*>(p) = make_float4(S[r][i][0], S[r][i][1], S[r][i][2], S[r][i][3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) if (c + e < dk) p[e] = S[r][i][e];
            }
        }
}

// ---------------------------------------------------------------------------------- chunks
// A chunk's tile in shared memory: CH rows of DP bfloat16, 16 bytes of padding each.
template <int DP> struct Tile {
    static constexpr int ROW = DP + 8;
    static constexpr int ELEMS = CH * ROW;
};
constexpr int DV = 64;                  // value channels of a unit
constexpr int PIECE = 16 * 16;          // floats of a piece of a state
__host__ __device__ constexpr int keys_padded(int dk) { return dk <= 64 ? 64 : 128; }
// pieces of one head's state: [units][keys / 16][4]
__host__ __device__ inline int pieces_of(int dk, int dv) { return (dv + DV - 1) / DV * (keys_padded(dk) / 16) * (DV / 16); }

// powers of two; what is below 2^-126 is zero
__device__ __forceinline__ float ds_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

struct ChunkAt { int row, n, slot; };       // first flat row, tokens, index among the step's chunks

// chunk c of request req, or n = 0. A request's chunks have the indices q_start / CH + req .. : enough room for every
// request's last, partly filled chunk.
__device__ __forceinline__ ChunkAt chunk_at(const int* __restrict__ q_start, int req, int c) {
    const int first = q_start[req], last = q_start[req + 1];
    const int row = first + c * CH;
    return {row, max(0, min(CH, last - row)), (first - q_start[0]) / CH + req + c};
}

// One warp: per token of the chunk (2 lane and 2 lane + 1 a lane) the sum of the decays' log2 up to it and the factor on its value;
// tokens that do not exist do not decay.
__device__ __forceinline__ void chunk_sums(const DsIn& in, const ChunkAt& at, int h, double (&sum)[2], float (&f)[2]) {
    const int lane = threadIdx.x & 31;
    const bool fixed = in.raw == nullptr;
    const float rate2 = fixed ? 0.f : expf(in.a_log[h]) * LOG2E, bias = fixed ? 0.f : in.bias[h];
    const float fixed2 = fixed ? fmaxf(in.log2_decay[h], NO_DECAY_LEFT) : 0.f;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int t = 2 * lane + e;
        float d = 0.f;
        f[e] = 0.f;
        if (t < at.n) {
            f[e] = fixed ? 1.0f : softplus(in.raw[(size_t)(at.row + t) * in.ld_raw + h] + bias);
            d = fixed ? fixed2 : fmaxf(-rate2 * f[e], NO_DECAY_LEFT);
        }
        sum[e] = (double)d;
    }
    sum[1] += sum[0];
    double before = sum[1];         // of this lane's tokens and all before them
#pragma unroll
    for (int m = 1; m < 32; m <<= 1) {
        const double x = __shfl_up_sync(0xffffffffu, before, m);
        if (lane >= m) before += x;
    }
    double up = __shfl_up_sync(0xffffffffu, before, 1);
    if (lane == 0) up = 0.0;
    sum[0] += up;
    sum[1] += up;
}

// The sums as two floats each, so that differences of them keep their digits.
__device__ __forceinline__ void chunk_decays(const DsIn& in, const ChunkAt& at, int h, float* hi_s, float* lo_s, float* f_s) {
    const int lane = threadIdx.x & 31;
    double sum[2];
    float f[2];
    chunk_sums(in, at, h, sum, f);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const float hi = (float)sum[e];
        hi_s[2 * lane + e] = hi;
        lo_s[2 * lane + e] = (float)(sum[e] - (double)hi);
        f_s[2 * lane + e] = f[e];
    }
}

// x and y as bfloat16 and as the bfloat16 of what that leaves out
__device__ __forceinline__ void split2(float x, float y, unsigned& hi, unsigned& lo) {
    hi = pack_bf16(x, y);
    lo = pack_bf16(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}

__device__ __forceinline__ void put4(__nv_bfloat16* p, const float4& x) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(x.x, x.y), pack_bf16(x.z, x.w));
}

__device__ __forceinline__ void ds_cp_async_16(void* smem, const void* gmem, bool valid) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(smem);
    const int n = valid ? 16 : 0;       // 0 source bytes: the destination is zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(d), "l"(gmem), "r"(n));
}
__device__ __forceinline__ void ds_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void ds_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }

// n rows of `src` (row stride ld, `width` elements from its column 0 on) into a tile; rows and columns that do not exist are zeros.
// vec: rows of T start on 16-byte boundaries and the width fills whole 16-byte groups.
template <typename T, int DP>
__device__ __forceinline__ void load_rows(__nv_bfloat16* tile, const T* __restrict__ src, int ld, int n, int width, bool silu, bool vec) {
    if (sizeof(T) == 2 && vec && !silu) {
        for (int i = threadIdx.x; i < CH * (DP / 8); i += DS_THREADS) {
            const int r = i / (DP / 8), c = (i % (DP / 8)) * 8;
            const bool ok = r < n && c < width;
            ds_cp_async_16(tile + r * Tile<DP>::ROW + c, ok ? src + (size_t)r * ld + c : src, ok);
        }
        return;
    }
#pragma unroll 8
    for (int i = threadIdx.x; i < CH * (DP / 4); i += DS_THREADS) {
        const int r = i / (DP / 4), c = (i % (DP / 4)) * 4;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (r < n) x = row4(src + (size_t)r * ld, c, width, vec);
        if (silu) silu4(x);
        put4(tile + r * Tile<DP>::ROW + c, x);
    }
}

// Where a block stands: a chunk of a request and U units that share q and k. grid: (chunks, units / U, requests). piece: the first
// of a unit's pieces of the chunk's state.
struct Unit { int h, v0, nv; size_t piece; };
__device__ __forceinline__ Unit unit_of(const DsIn& in, const ChunkAt& at, int u) {
    const int per_head = (in.dv + DV - 1) / DV, h = u / per_head, v0 = (u % per_head) * DV;
    return {h, v0, min(DV, in.dv - v0), ((size_t)at.slot * in.heads + h) * pieces_of(in.dk, in.dv) + v0 / 16 * (keys_padded(in.dk) / 16)};
}

// What a chunk adds to a zero state: local[chunk, head, piece], and the chunk's whole decay. A warp owns 16
// value channels: rows of the product (weighted v)^T . k over the chunk's tokens; the weights go on v in registers, in 32-bit.
template <typename T, int DKP, int U>
__global__ void __launch_bounds__(DS_THREADS, 5)
chunk_state_kernel(const DsIn in, float* __restrict__ local, float* __restrict__ decays) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ __align__(16) float w_s[U][CH];      // what a token's value is multiplied with: its factor and the decays behind it
    pdl_launch_dependents();
    pdl_wait();
    const ChunkAt at = chunk_at(in.q_start, blockIdx.z, blockIdx.x);
    if (at.n == 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mat = lane >> 3, rr = lane & 7, t = lane & 3, u0 = blockIdx.y * U;
    constexpr int RK = Tile<DKP>::ROW, RV = Tile<DV>::ROW;
    __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(smem);
    __nv_bfloat16* v_s = k_s + Tile<DKP>::ELEMS;
    load_rows<T, DKP>(k_s, in.k_at<T>(at.row, unit_of(in, at, u0).h / (in.heads / in.kq_heads)), in.ldk, at.n, in.dk, in.silu != 0, in.vec != 0);
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const Unit b = unit_of(in, at, u0 + u);
        load_rows<T, DV>(v_s + u * Tile<DV>::ELEMS, in.v_at<T>(at.row, b.h) + b.v0, in.ldv, at.n, b.nv, in.silu != 0, in.vec != 0);
    }
    ds_commit();
    if (warp < U) {
        const Unit b = unit_of(in, at, u0 + warp);
        double sum[2];
        float f[2];
        chunk_sums(in, at, b.h, sum, f);
        const double end = __shfl_sync(0xffffffffu, sum[1], 31);
        *reinterpret_cast<float2*>(&w_s[warp][2 * lane]) = make_float2(ds_exp2((float)(end - sum[0])) * f[0], ds_exp2((float)(end - sum[1])) * f[1]);
        if (lane == 0 && b.v0 == 0) decays[(size_t)at.slot * in.heads + b.h] = ds_exp2((float)end);
    }
    ds_wait<0>();
    __syncthreads();
#pragma unroll 1
    for (int u = 0; u < U; ++u) {
        const Unit b = unit_of(in, at, u0 + u);
        float acc[DKP / 8][4];
#pragma unroll
        for (int n = 0; n < DKP / 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
#pragma unroll 1      // (unrolled, the kernel waits for its own instructions: they run once a block)
        for (int kb = 0; kb < CH / 16; ++kb) {
            unsigned a[4], a_hi[4], a_lo[4];       // A: value channel x token, out of [token][value channel]
            ldmatrix_x4_trans(a, v_s + u * Tile<DV>::ELEMS + (kb * 16 + (mat >> 1) * 8 + rr) * RV + warp * 16 + (mat & 1) * 8);
#pragma unroll
            for (int half = 0; half < 2; ++half) {      // the thread's tokens: 2t, 2t + 1 of eight
                const float2 w = *reinterpret_cast<const float2*>(&w_s[u][kb * 16 + half * 8 + 2 * t]);
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a[2 * half + r]));
                    split2(v.x * w.x, v.y * w.y, a_hi[2 * half + r], a_lo[2 * half + r]);
                }
            }
#pragma unroll
            for (int np = 0; np < DKP / 16; ++np) {     // B: token x key channel
                unsigned bk[4];
                ldmatrix_x4_trans(bk, k_s + (kb * 16 + (mat & 1) * 8 + rr) * RK + np * 16 + (mat >> 1) * 8);
                mma_bf16(acc[2 * np], a_hi, bk[0], bk[1]);
                mma_bf16(acc[2 * np + 1], a_hi, bk[2], bk[3]);
                mma_bf16(acc[2 * np], a_lo, bk[0], bk[1]);
                mma_bf16(acc[2 * np + 1], a_lo, bk[2], bk[3]);
            }
        }
        float* out = local + (b.piece + warp) * PIECE + lane * 8;       // (zeros where the head has fewer channels)
#pragma unroll
        for (int kk = 0; kk < DKP / 16; ++kk) {
            float4* to = reinterpret_cast<float4*>(out + kk * 4 * PIECE);
            to[0] = make_float4(acc[2 * kk][0], acc[2 * kk][1], acc[2 * kk + 1][0], acc[2 * kk + 1][1]);
            to[1] = make_float4(acc[2 * kk][2], acc[2 * kk][3], acc[2 * kk + 1][2], acc[2 * kk + 1][3]);
        }
    }
}

// local[chunk] (what the chunk adds) becomes the chunk's entry state; the slot's state moves past the request's last chunk. A thread
// per lane of a piece; the chunks' loads run ahead of the chain. The entry states are written as the products read them: a lane's
// eight bfloat16 and then the bfloat16 of their remainders where its eight floats were.
__global__ void __launch_bounds__(128)
chunk_chain_kernel(float* __restrict__ state, long long state_ld, int state_off, const int* __restrict__ q_start, const int* __restrict__ slots,
                   float* __restrict__ local, const float* __restrict__ decays, int heads, int dk, int dv) {
    constexpr int AHEAD = 8;
    pdl_launch_dependents();
    pdl_wait();
    const int req = blockIdx.y, pieces = pieces_of(dk, dv), per_keys = keys_padded(dk) / 16;
    const long long w = (long long)blockIdx.x * 4 + (threadIdx.x >> 5), all = (long long)heads * pieces;
    const int len = q_start[req + 1] - q_start[req], chunks = (len + CH - 1) / CH;
    if (w >= all || chunks == 0) return;
    const int lane = threadIdx.x & 31, h = (int)(w / pieces), piece = (int)(w % pieces), slot0 = (q_start[req] - q_start[0]) / CH + req;
    const int j0 = piece / (4 * per_keys) * DV + piece % 4 * 16 + (lane >> 2), c0 = piece / 4 % per_keys * 16 + 2 * (lane & 3);
    float* st = state + (long long)slots[req] * state_ld + state_off + (long long)h * dv * dk;
    float* at = local + ((size_t)slot0 * all + w) * PIECE + lane * 8;
    const size_t step = (size_t)all * PIECE;
    const float* dec = decays + (size_t)slot0 * heads + h;
    float S[8];
#pragma unroll
    for (int n = 0; n < 8; ++n) {
        const int j = j0 + (n & 4) * 2, c = c0 + (n & 2) * 4 + (n & 1);
        S[n] = j < dv && c < dk ? st[(long long)j * dk + c] : 0.f;
    }
    for (int k0 = 0; k0 < chunks; k0 += AHEAD) {
        float4 x[AHEAD][2];
        float d[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (k0 + i < chunks) {
                const float4* from = reinterpret_cast<const float4*>(at + (size_t)(k0 + i) * step);
                x[i][0] = from[0];
                x[i][1] = from[1];
                d[i] = dec[(size_t)(k0 + i) * heads];
            }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (k0 + i < chunks) {
                uint4* to = reinterpret_cast<uint4*>(at + (size_t)(k0 + i) * step);
                unsigned hi[4], lo[4];
#pragma unroll
                for (int n = 0; n < 4; ++n) split2(S[2 * n], S[2 * n + 1], hi[n], lo[n]);
                to[0] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                to[1] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
                const float add[8] = {x[i][0].x, x[i][0].y, x[i][0].z, x[i][0].w, x[i][1].x, x[i][1].y, x[i][1].z, x[i][1].w};
#pragma unroll
                for (int n = 0; n < 8; ++n) S[n] = fmaf(d[i], S[n], add[n]);
            }
    }
#pragma unroll
    for (int n = 0; n < 8; ++n) {
        const int j = j0 + (n & 4) * 2, c = c0 + (n & 2) * 4 + (n & 1);
        if (j < dv && c < dk) st[(long long)j * dk + c] = S[n];
    }
}

// The outputs of a chunk from its entry state. A warp owns 16 tokens; what q . k gives serves all of the block's units.
template <typename T, int DKP, int U>
__global__ void __launch_bounds__(DS_THREADS, U == 1 ? 5 : 4)
chunk_output_kernel(const DsIn in, const float* __restrict__ entry, float* __restrict__ o, int ldo) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ __align__(16) float hi_s[U][CH], lo_s[U][CH], f_s[U][CH];
    pdl_launch_dependents();
    pdl_wait();
    const ChunkAt at = chunk_at(in.q_start, blockIdx.z, blockIdx.x);
    if (at.n == 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mat = lane >> 3, rr = lane & 7, g = lane >> 2, t4 = lane & 3, u0 = blockIdx.y * U;
    constexpr int RK = Tile<DKP>::ROW, RV = Tile<DV>::ROW;
    __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem);
    __nv_bfloat16* k_s = q_s + Tile<DKP>::ELEMS;
    __nv_bfloat16* v_s = k_s + Tile<DKP>::ELEMS;
    const bool vec = in.vec != 0, silu = in.silu != 0;
    const int hq = unit_of(in, at, u0).h / (in.heads / in.kq_heads);
    load_rows<T, DKP>(q_s, in.q_at<T>(at.row, hq), in.ldq, at.n, in.dk, silu, vec);
    ds_commit();
    load_rows<T, DKP>(k_s, in.k_at<T>(at.row, hq), in.ldk, at.n, in.dk, silu, vec);
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const Unit b = unit_of(in, at, u0 + u);
        load_rows<T, DV>(v_s + u * Tile<DV>::ELEMS, in.v_at<T>(at.row, b.h) + b.v0, in.ldv, at.n, b.nv, silu, vec);
    }
    ds_commit();
    if (warp < U) chunk_decays(in, at, unit_of(in, at, u0 + warp).h, hi_s[warp], lo_s[warp], f_s[warp]);
    ds_wait<1>();
    __syncthreads();
    Unit b[U];
#pragma unroll
    for (int u = 0; u < U; ++u) b[u] = unit_of(in, at, u0 + u);
    const __nv_bfloat16* q_w = q_s + (warp * 16 + (mat & 1) * 8 + rr) * RK + (mat >> 1) * 8;
    float acc[U][DV / 8][4];
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
        for (int n = 0; n < DV / 8; ++n) acc[u][n][0] = acc[u][n][1] = acc[u][n][2] = acc[u][n][3] = 0.f;
    // q . S_in. (The loops over keys stay loops: unrolled, the kernel waits for its own instructions, which run once a block.)
#pragma unroll 1
    for (int kk = 0; kk < DKP / 16; ++kk) {
        unsigned q[4];
        ldmatrix_x4(q, q_w + kk * 16);
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const uint4* piece = reinterpret_cast<const uint4*>(entry + (b[u].piece + kk * 4) * PIECE + lane * 8);      // the state's bfloat16, then its remainders
#pragma unroll
            for (int np = 0; np < DV / 16; ++np) {
                const uint4 bh = piece[np * (PIECE / 4)], bl = piece[np * (PIECE / 4) + 1];
                mma_bf16(acc[u][2 * np], q, bh.x, bh.y);
                mma_bf16(acc[u][2 * np + 1], q, bh.z, bh.w);
                mma_bf16(acc[u][2 * np], q, bl.x, bl.y);
                mma_bf16(acc[u][2 * np + 1], q, bl.z, bl.w);
            }
        }
    }
    float t_hi[U][2], t_lo[U][2];
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            t_hi[u][r] = hi_s[u][warp * 16 + g + 8 * r];
            t_lo[u][r] = lo_s[u][warp * 16 + g + 8 * r];
            const float w = ds_exp2(t_hi[u][r] + t_lo[u][r]);
#pragma unroll
            for (int n = 0; n < DV / 8; ++n) { acc[u][n][2 * r] *= w; acc[u][n][2 * r + 1] *= w; }
        }
    ds_wait<0>();
    __syncthreads();
    if (warp * 16 >= at.n) return;
    // the chunk's own tokens, 16 keys at a time up to the warp's last token; what q . k gives serves all units
#pragma unroll 1
    for (int kb = 0; kb <= warp; ++kb) {
        float s[2][4] = {};
        const __nv_bfloat16* k_w = k_s + (kb * 16 + (mat >> 1) * 8 + rr) * RK + (mat & 1) * 8;
#pragma unroll 2
        for (int kk = 0; kk < DKP / 16; ++kk) {
            unsigned q[4], bk[4];
            ldmatrix_x4(q, q_w + kk * 16);
            ldmatrix_x4(bk, k_w + kk * 16);
            mma_bf16(s[0], q, bk[0], bk[1]);
            mma_bf16(s[1], q, bk[2], bk[3]);
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            unsigned p_hi[4], p_lo[4];
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const int key = kb * 16 + n * 8 + 2 * t4;
                const float2 k_hi = *reinterpret_cast<const float2*>(&hi_s[u][key]), k_lo = *reinterpret_cast<const float2*>(&lo_s[u][key]);
                const float2 f = *reinterpret_cast<const float2*>(&f_s[u][key]);
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    const int tok = warp * 16 + g + 8 * r;
                    const float w0 = ds_exp2((t_hi[u][r] - k_hi.x) + (t_lo[u][r] - k_lo.x)) * f.x, w1 = ds_exp2((t_hi[u][r] - k_hi.y) + (t_lo[u][r] - k_lo.y)) * f.y;
                    const float x0 = key <= tok ? s[n][2 * r] * w0 : 0.f, x1 = key + 1 <= tok ? s[n][2 * r + 1] * w1 : 0.f;
                    split2(x0, x1, p_hi[2 * n + r], p_lo[2 * n + r]);
                }
            }
#pragma unroll
            for (int np = 0; np < DV / 16; ++np) {
                unsigned bv[4];
                ldmatrix_x4_trans(bv, v_s + u * Tile<DV>::ELEMS + (kb * 16 + (mat & 1) * 8 + rr) * RV + np * 16 + (mat >> 1) * 8);
                mma_bf16(acc[u][2 * np], p_hi, bv[0], bv[1]);
                mma_bf16(acc[u][2 * np + 1], p_hi, bv[2], bv[3]);
                mma_bf16(acc[u][2 * np], p_lo, bv[0], bv[1]);
                mma_bf16(acc[u][2 * np + 1], p_lo, bv[2], bv[3]);
            }
        }
    }
    const bool pairs = in.dv % 2 == 0 && ldo % 2 == 0 && ((uintptr_t)o & 7) == 0;
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int tok = warp * 16 + g + 8 * r;
            if (tok >= at.n) continue;
            float* row = o + (size_t)(at.row + tok) * ldo + (size_t)b[u].h * in.dv + b[u].v0;
#pragma unroll
            for (int n = 0; n < DV / 8; ++n) {
                const int c = n * 8 + 2 * t4;
                if (pairs) {
                    if (c < b[u].nv) *reinterpret_cast<float2*>(row + c) = make_float2(acc[u][n][2 * r], acc[u][n][2 * r + 1]);
                } else {
                    if (c < b[u].nv) row[c] = acc[u][n][2 * r];
                    if (c + 1 < b[u].nv) row[c + 1] = acc[u][n][2 * r + 1];
                }
            }
        }
}

template <typename T, int DKP, int U>
int launch_chunks(const DsIn& in, float* state, long long state_ld, int state_off, float* o, int ldo, int n_req, int max_len, float* local,
                  float* decays, cudaStream_t stream) {
    constexpr int SMEM_STATE = (Tile<DKP>::ELEMS + U * Tile<DV>::ELEMS) * 2, SMEM_OUT = (2 * Tile<DKP>::ELEMS + U * Tile<DV>::ELEMS) * 2;
    static bool configured = false;
    if (!configured) {
        NIB_CUDA(cudaFuncSetAttribute(chunk_state_kernel<T, DKP, U>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_STATE));
        NIB_CUDA(cudaFuncSetAttribute(chunk_output_kernel<T, DKP, U>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_OUT));
        configured = true;
    }
    const dim3 grid(ceil_div(max_len, CH), in.heads * ceil_div(in.dv, DV) / U, n_req);
    NIB_CUDA(launch_pdl(chunk_state_kernel<T, DKP, U>, grid, dim3(DS_THREADS), (size_t)SMEM_STATE, stream, in, local, decays));
    NIB_CUDA(launch_pdl(chunk_chain_kernel, dim3(ceil_div((long long)in.heads * pieces_of(in.dk, in.dv), 4), n_req), dim3(128), (size_t)0, stream, state,
                        state_ld, state_off, in.q_start, in.slots, local, (const float*)decays, in.heads, in.dk, in.dv));
    NIB_CUDA(launch_pdl(chunk_output_kernel<T, DKP, U>, grid, dim3(DS_THREADS), (size_t)SMEM_OUT, stream, in, (const float*)local, o, ldo));
    NIB_LAUNCH_CHECK();
    return 0;
}

template <typename T, int LANES, int NV>
int launch_step(const DsIn& in, float* state, long long state_ld, int state_off, float* o, int ldo, int n_req, cudaStream_t stream) {
    const dim3 grid(ceil_div(in.dv, (DS_THREADS / LANES) * R), in.heads, n_req);
    NIB_CUDA(launch_pdl(decay_step_kernel<T, LANES, NV>, grid, dim3(DS_THREADS), (size_t)0, stream, in, state, state_ld, state_off, o, ldo));
    NIB_LAUNCH_CHECK();
    return 0;
}

template <typename T>
int scan(DsIn in, float* state, long long state_ld, int state_off, float* o, int ldo, int tokens, int n_req, int max_len, float* scratch,
         cudaStream_t stream) {
    const int dk = in.dk, dv = in.dv;
    if (scratch == nullptr) {       // four elements a load
        auto aligned = [](const void* p, long long ld) { return ((uintptr_t)p & (4 * sizeof(T) - 1)) == 0 && ld % 4 == 0; };
        in.vec = dk % 4 == 0 && aligned(in.q, in.ldq) && aligned(in.k, in.ldk) && ((uintptr_t)state & 15) == 0 && state_ld % 4 == 0 && state_off % 4 == 0;
        if (dk <= 32) return launch_step<T, 8, 1>(in, state, state_ld, state_off, o, ldo, n_req, stream);
        if (dk <= 64) return launch_step<T, 16, 1>(in, state, state_ld, state_off, o, ldo, n_req, stream);
        if (dk <= 128) return launch_step<T, 32, 1>(in, state, state_ld, state_off, o, ldo, n_req, stream);
        return launch_step<T, 32, 2>(in, state, state_ld, state_off, o, ldo, n_req, stream);
    }
    constexpr int G = 16 / sizeof(T);       // 16 bytes a load
    auto aligned = [](const void* p, long long ld) { return ((uintptr_t)p & 15) == 0 && ld % G == 0; };
    in.vec = dk % G == 0 && dv % G == 0 && aligned(in.q, in.ldq) && aligned(in.k, in.ldk) && aligned(in.v, in.ldv);
    float* decays = scratch + ((long long)tokens / CH + n_req) * in.heads * pieces_of(dk, dv) * PIECE;
    // pairs of units of heads with the same q and k, once their blocks fill the GPU
    const int sharing = in.heads / in.kq_heads * ceil_div(dv, DV);
    const bool two = sharing % 2 == 0 && (long long)in.heads * ceil_div(dv, DV) * ceil_div(tokens, CH) >= 4LL * 148;
#define NIB_DS(DKP, U) launch_chunks<T, DKP, U>(in, state, state_ld, state_off, o, ldo, n_req, max_len, scratch, decays, stream)
    if (dk <= 64) return two ? NIB_DS(64, 2) : NIB_DS(64, 1);
    return two ? NIB_DS(128, 2) : NIB_DS(128, 1);
#undef NIB_DS
}

}  // namespace

// Floats of scratch for a step of `tokens` tokens of n_req requests in chunks: entry states, then decays.
NIB_API long long nib_decay_state_scratch(long long tokens, int n_req, int heads, int dk, int dv) {
    const long long slots = tokens / CH + n_req;
    return slots * heads * pieces_of(dk, dv) * PIECE + slots * heads;
}

NIB_API int nib_decay_state_chunks_supported(int dk, int dv) { return dk > 0 && dv > 0 && dk <= 128 ? 1 : 0; }

// q, k and v of `dtype`. q_start [n_req + 1] and slots [n_req] of the requests taken here (rows are counted from the step's first one).
// scratch null: token by token; else in chunks, with nib_decay_state_scratch floats for the requests' tokens.
NIB_API int nib_decay_state_scan(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, const float* raw, int ld_raw,
                                 const float* bias, const float* a_log, const float* decay, const float* log2_decay, int silu, float* state,
                                 long long state_ld, int state_off, const int* q_start, const int* slots, float* o, int ldo, int tokens, int n_req,
                                 int max_len, int heads, int kq_heads, int dk, int dv, int dtype, float* scratch, cudaStream_t stream) {
    NIB_REQUIRE(heads > 0 && kq_heads > 0 && heads % kq_heads == 0, "decay_state_scan: %d heads do not share %d key heads", heads, kq_heads);
    NIB_REQUIRE(dk > 0 && dk <= 256 && dv > 0, "decay_state_scan: key size %d is outside 1..256", dk);
    NIB_REQUIRE(raw != nullptr ? (bias != nullptr && a_log != nullptr) : (decay != nullptr && log2_decay != nullptr),
                "decay_state_scan: step sizes need bias and a_log, fixed decays their logarithms");
    NIB_REQUIRE(n_req >= 0 && n_req <= 65535 && (long long)heads * ceil_div(dv, DV) <= 65535 && max_len >= 0, "decay_state_scan: bad counts");
    NIB_REQUIRE(((uintptr_t)scratch & 15) == 0, "decay_state_scan: scratch must start on a 16-byte boundary");
    NIB_REQUIRE(scratch == nullptr || nib_decay_state_chunks_supported(dk, dv) == 1, "decay_state_scan: chunks take keys up to 128, not %d", dk);
    if (n_req == 0 || max_len == 0) return 0;
    const DsIn in{q, k, v, raw, bias, a_log, decay, log2_decay, q_start, slots, ldq, ldk, ldv, ld_raw, heads, kq_heads, dk, dv, silu, 0};
    if (dtype == NIB_F32) return scan<float>(in, state, state_ld, state_off, o, ldo, tokens, n_req, max_len, scratch, stream);
    NIB_REQUIRE(dtype == NIB_BF16, "decay_state_scan: unknown dtype %d", dtype);
    return scan<__nv_bfloat16>(in, state, state_ld, state_off, o, ldo, tokens, n_req, max_len, scratch, stream);
}
