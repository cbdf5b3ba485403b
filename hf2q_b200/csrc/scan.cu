// Recurrent mixers with a matrix state per head, token after token in 32-bit arithmetic:
//
//   mlstm   exponential input / forget gates with a running maximum (matrix memory of xLSTM)
//   delta   gated delta rule, one decay per head and key channel
//   ssd     scalar decay per head and token (Mamba-2)
//
// All keep S[key channel][value column] and treat a value column independently, so the state lives in registers:
// sixteen lanes share a column (each holds key channels 32 c + 2 l and + 1), a warp carries two columns, a CTA of eight
// warps sixteen columns of one head: the token chain is latency-bound, so many short warps beat few long ones.  A token costs no block barrier; sums over the key channels are four shuffles.
// Tokens are staged in shared memory in batches by asynchronous copies, two batches in flight.  The state in memory
// is [head][column][key channel, padded to 32] (f32), which makes a lane's channels consecutive.
#include <math_constants.h>

#include "seq_common.cuh"

namespace hf2q {
namespace {
using namespace seq;

constexpr int SC_WARPS = 8, SC_COLS = 16, SC_TB = 16, SC_THREADS = SC_WARPS * 32;

__device__ __forceinline__ float group_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    v += __shfl_xor_sync(0xffffffffu, v, 4);
    v += __shfl_xor_sync(0xffffffffu, v, 8);
    return v;
}
// Sums of sixteen values over the sixteen lanes of a group, transposed: lane l ends with the sum of v[l] (15 shuffles).
__device__ __forceinline__ float group_transpose_sum(float (&v)[16], uint32_t l) {
#pragma unroll
    for (int w = 8; w > 0; w >>= 1) {
        const bool up = l & w;
#pragma unroll
        for (int i = 0; i < w; ++i) {
            const float other = __shfl_xor_sync(0xffffffffu, up ? v[i] : v[i + w], w);
            v[i] = (up ? v[i + w] : v[i]) + other;
        }
    }
    return v[0];
}
// rows of `count` floats -> shared memory, asynchronously, 16 bytes at a time where both sides allow it; a warp takes
// whole rows
__device__ __forceinline__ void stage_rows(float* dst, uint32_t dst_ld, const float* src, size_t src_ld, uint32_t rows, uint32_t count) {
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (count % 4 == 0 && src_ld % 4 == 0 && dst_ld % 4 == 0 && (reinterpret_cast<uintptr_t>(src) & 15) == 0) {
        for (uint32_t r = warp; r < rows; r += SC_WARPS)
            for (uint32_t c = 4 * lane; c < count; c += 128) cp_async16(dst + r * dst_ld + c, src + r * src_ld + c);
    } else {
        for (uint32_t r = warp; r < rows; r += SC_WARPS)
            for (uint32_t c = lane; c < count; c += 32) cp_async4(dst + r * dst_ld + c, src + r * src_ld + c);
    }
}

// two f32 values in a 64-bit register; one instruction works on both (IEEE arithmetic on each half)
typedef unsigned long long f2;
__device__ __forceinline__ f2 f2_mul(f2 a, f2 b) { f2 d; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }
__device__ __forceinline__ f2 f2_fma(f2 a, f2 b, f2 c) { f2 d; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c)); return d; }
__device__ __forceinline__ f2 f2_add(f2 a, f2 b) { f2 d; asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }
__device__ __forceinline__ f2 f2_both(float a) { f2 d; asm("mov.b64 %0, {%1, %1};" : "=l"(d) : "f"(a)); return d; }
__device__ __forceinline__ float f2_sum(f2 a) { float x, y; asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a)); return x + y; }

template <int RQ> struct Vec {                       // a lane's RQ pairs of key channels
    f2 v[RQ];
    __device__ __forceinline__ void load(const float* p) {
#pragma unroll
        for (int c = 0; c < RQ; ++c) v[c] = *reinterpret_cast<const f2*>(p + 32 * c);
    }
    __device__ __forceinline__ void zero() {
#pragma unroll
        for (int c = 0; c < RQ; ++c) v[c] = 0ull;
    }
    __device__ __forceinline__ void store(float* p) const {
#pragma unroll
        for (int c = 0; c < RQ; ++c) *reinterpret_cast<f2*>(p + 32 * c) = v[c];
    }
    // sum over this lane's channels, in two interleaved pairs of partial sums
    __device__ __forceinline__ float dot(const Vec& k) const {
        f2 s[2] = {f2_mul(v[0], k.v[0]), 0ull};
#pragma unroll
        for (int c = 1; c < RQ; ++c) s[c & 1] = f2_fma(v[c], k.v[c], s[c & 1]);
        return f2_sum(RQ > 1 ? f2_add(s[0], s[1]) : s[0]);
    }
    __device__ __forceinline__ void scale(const Vec& k) {
#pragma unroll
        for (int c = 0; c < RQ; ++c) v[c] = f2_mul(v[c], k.v[c]);
    }
    __device__ __forceinline__ void axpy(const Vec& k, float a) {
        const f2 aa = f2_both(a);
#pragma unroll
        for (int c = 0; c < RQ; ++c) v[c] = f2_fma(k.v[c], aa, v[c]);
    }
    __device__ __forceinline__ void decay_axpy(float keep, const Vec& k, float a) {
        const f2 kk = f2_both(keep), aa = f2_both(a);
#pragma unroll
        for (int c = 0; c < RQ; ++c) v[c] = f2_fma(kk, v[c], f2_mul(k.v[c], aa));
    }
};

// ---------------------------------------------------------------- mLSTM
template <int RQ>
__global__ void __launch_bounds__(SC_THREADS) mlstm_kernel(const __grid_constant__ hf2q_mlstm a, uint32_t m, float* __restrict__ out) {
    constexpr uint32_t DP = 32 * RQ;
    extern __shared__ __align__(16) float dsm[];                    // k, q: [2][SC_TB][DP] each
    float* ks = dsm;
    float* qs = dsm + 2 * SC_TB * DP;
    __shared__ __align__(16) float vs[2][SC_TB][SC_COLS];
    __shared__ float gk[2][SC_TB], gw[2][SC_TB], ge[2][SC_TB];     // keep, write, exp(-maximum)
    pdl_trigger();
    pdl_wait();
    const uint32_t h = blockIdx.x, slice = blockIdx.y, n_slices = gridDim.y;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lg = lane & 15;
    const uint32_t col_s = warp * 2 + (lane >> 4), col0 = slice * SC_COLS, col = col0 + col_s;
    const uint32_t n_cols = min(static_cast<uint32_t>(SC_COLS), a.vdim - col0);
    const bool live = col < a.vdim;
    const float q_scale = 1.0f / sqrtf(static_cast<float>(a.dim));
    float* mp = a.mx + static_cast<size_t>(h) * n_slices + slice;
    float mx = *mp;                                          // carried by the last warp
    // channels past dim stay zero in shared memory, so the padded part of the state stays zero too
    for (uint32_t i = threadIdx.x; i < 4 * SC_TB * DP; i += SC_THREADS) dsm[i] = 0.f;
    for (uint32_t i = threadIdx.x; i < 2 * SC_TB * SC_COLS; i += SC_THREADS) (&vs[0][0][0])[i] = 0.f;
    __syncthreads();
    auto stage = [&](uint32_t t0, uint32_t b) {
        const uint32_t n = min(static_cast<uint32_t>(SC_TB), m - t0);
        const float* row = a.proj + static_cast<size_t>(t0) * a.ld;
        stage_rows(ks + b * SC_TB * DP, DP, row + a.k_off + h * a.dim, a.ld, n, a.dim);
        stage_rows(qs + b * SC_TB * DP, DP, row + a.q_off + h * a.dim, a.ld, n, a.dim);
        stage_rows(vs[b][0], SC_COLS, row + a.v_off + h * a.vdim + col0, a.ld, n, n_cols);
        // gate factors of the batch, by the last warp (lane = token): the running maximum is a max-plus scan over the
        // pairs (f, i), m_t = max(m + f_1 + .. + f_t, max_s (i_s + f_(s+1) + .. + f_t))
        if (warp == SC_WARPS - 1) {
            float f = 0.f, x = -CUDART_INF_F;
            if (lane < n) {
                const float* g = row + static_cast<size_t>(lane) * a.ld + h;
                x = a.gate_cap * tanhf((g[a.i_off] + a.i_bias[h]) / a.gate_cap);
                f = -softplusf(-a.gate_cap * tanhf((g[a.f_off] + a.f_bias[h]) / a.gate_cap));
            }
            const float f_own = f, x_own = x;
#pragma unroll
            for (int d = 1; d < SC_TB; d *= 2) {
                const float fo = __shfl_up_sync(0xffffffffu, f, d), xo = __shfl_up_sync(0xffffffffu, x, d);
                if (lane >= d) { x = fmaxf(xo + f, x); f += fo; }
            }
            const float m_t = fmaxf(mx + f, x);
            float before = __shfl_up_sync(0xffffffffu, m_t, 1);
            if (lane == 0) before = mx;
            if (lane < n) {
                gk[b][lane] = expf(f_own + before - m_t);
                gw[b][lane] = expf(x_own - m_t);
                ge[b][lane] = expf(-m_t);
            }
            mx = __shfl_sync(0xffffffffu, m_t, n - 1);
        }
        cp_async_commit();
    };
    Vec<RQ> S, N;
    float* sp = a.s + (static_cast<size_t>(h) * a.vdim + (live ? col : 0)) * DP + 2 * lg;
    float* np = a.n + (static_cast<size_t>(h) * n_slices + slice) * DP + 2 * lg;
    if (live) S.load(sp); else S.zero();
    N.load(np);
    stage(0, 0);
    for (uint32_t t0 = 0, b = 0; t0 < m; t0 += SC_TB, b ^= 1) {
        if (t0 + SC_TB < m) { stage(t0 + SC_TB, b ^ 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        const uint32_t n = min(static_cast<uint32_t>(SC_TB), m - t0);
        // a token's operands are read one token ahead of their use
        struct Operands { Vec<RQ> k, q; float keep, write, v; };
        auto fetch = [&](uint32_t j) {
            Operands t;
            t.k.load(ks + (b * SC_TB + j) * DP + 2 * lg);
            t.q.load(qs + (b * SC_TB + j) * DP + 2 * lg);
            t.keep = gk[b][j];
            t.write = gw[b][j];
            t.v = vs[b][j][col_s];
            return t;
        };
        auto token = [&](const Operands& t, float& num, float& den) {      // this lane's part of both sums
            S.decay_axpy(t.keep, t.k, t.write * t.v);
            N.decay_axpy(t.keep, t.k, t.write);
            num = S.dot(t.q);
            den = N.dot(t.q);
        };
        auto finish = [&](uint32_t j, float num, float den) {
            if (live)
                out[static_cast<size_t>(t0 + j) * a.heads * a.vdim + static_cast<size_t>(h) * a.vdim + col] = num * q_scale / (fmaxf(fabsf(den * q_scale), ge[b][j]) + 1e-6f);
        };
        uint32_t j0 = 0;
        for (; j0 + 16 <= n; j0 += 16) {                     // sixteen tokens without a branch; lane i of a group finishes token i
            float num[16], den[16];
            Operands t = fetch(j0);
#pragma unroll
            for (uint32_t u = 0; u < 16; ++u) {
                const Operands next = fetch(j0 + (u < 15 ? u + 1 : 15));
                token(t, num[u], den[u]);
                t = next;
            }
            const float x = group_transpose_sum(num, lg), y = group_transpose_sum(den, lg);
            finish(j0 + lg, x, y);
        }
        for (; j0 < n; ++j0) {
            float x, y;
            token(fetch(j0), x, y);
            x = group_sum(x);
            y = group_sum(y);
            if (lg == 0) finish(j0, x, y);
        }
        __syncthreads();
    }
    if (live) S.store(sp);
    if (warp == 0 && lane < 16) N.store(np);
    if (warp == SC_WARPS - 1 && lane == 0) *mp = mx;
}

// ---------------------------------------------------------------- gated delta rule
// S <- g S;  u = beta (v - S^T k);  S <- S + k u;  o = S^T q
template <int RQ>
struct DeltaOperands {
    Vec<RQ> g, k, q;
    float v, beta;
};
template <int RQ>
__device__ __forceinline__ float delta_token(Vec<RQ>& S, const DeltaOperands<RQ>& t) {          // this lane's part of o
    S.scale(t.g);
    const float u = t.beta * (t.v - group_sum(S.dot(t.k)));
    S.axpy(t.k, u);
    return S.dot(t.q);
}

template <int RQ>
__global__ void __launch_bounds__(SC_THREADS) delta_scan_kernel(const __grid_constant__ hf2q_delta a, uint32_t m, const float* __restrict__ qkv,
                                                                const float* __restrict__ beta, const float* __restrict__ g, float* __restrict__ out) {
    constexpr uint32_t DP = 32 * RQ;
    extern __shared__ __align__(16) float dsm[];                    // k, q, g: [2][SC_TB][DP] each
    float* ks = dsm;
    float* qs = dsm + 2 * SC_TB * DP;
    float* gs = dsm + 4 * SC_TB * DP;
    __shared__ __align__(16) float vs[2][SC_TB][SC_COLS];
    __shared__ float bs[2][SC_TB];
    pdl_trigger();
    pdl_wait();
    const uint32_t h = blockIdx.x, slice = blockIdx.y, kvh = h / (a.heads / a.kv_heads);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lg = lane & 15;
    const uint32_t col_s = warp * 2 + (lane >> 4), col0 = slice * SC_COLS, col = col0 + col_s;
    const uint32_t n_cols = min(static_cast<uint32_t>(SC_COLS), a.vdim - col0);
    const bool live = col < a.vdim;
    const uint32_t qk = a.kv_heads * a.dim, ld = 2 * qk + a.heads * a.vdim;
    for (uint32_t i = threadIdx.x; i < 6 * SC_TB * DP; i += SC_THREADS) dsm[i] = 0.f;
    for (uint32_t i = threadIdx.x; i < 2 * SC_TB * SC_COLS; i += SC_THREADS) (&vs[0][0][0])[i] = 0.f;
    __syncthreads();
    auto stage = [&](uint32_t t0, uint32_t b) {
        const uint32_t n = min(static_cast<uint32_t>(SC_TB), m - t0);
        const float* row = qkv + static_cast<size_t>(t0) * ld;
        stage_rows(qs + b * SC_TB * DP, DP, row + kvh * a.dim, ld, n, a.dim);
        stage_rows(ks + b * SC_TB * DP, DP, row + qk + kvh * a.dim, ld, n, a.dim);
        stage_rows(vs[b][0], SC_COLS, row + 2 * qk + h * a.vdim + col0, ld, n, n_cols);
        stage_rows(gs + b * SC_TB * DP, DP, g + (static_cast<size_t>(t0) * a.heads + h) * a.dim, static_cast<size_t>(a.heads) * a.dim, n, a.dim);
        if (threadIdx.x < n) bs[b][threadIdx.x] = beta[static_cast<size_t>(t0 + threadIdx.x) * a.heads + h];
        cp_async_commit();
    };
    Vec<RQ> S;
    float* sp = a.s + (static_cast<size_t>(h) * a.vdim + (live ? col : 0)) * DP + 2 * lg;
    if (live) S.load(sp); else S.zero();
    stage(0, 0);
    for (uint32_t t0 = 0, b = 0; t0 < m; t0 += SC_TB, b ^= 1) {
        if (t0 + SC_TB < m) { stage(t0 + SC_TB, b ^ 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        const uint32_t n = min(static_cast<uint32_t>(SC_TB), m - t0);
        auto fetch = [&](uint32_t j) {                       // read one token ahead of their use
            const uint32_t o = (b * SC_TB + j) * DP + 2 * lg;
            DeltaOperands<RQ> t;
            t.g.load(gs + o);
            t.k.load(ks + o);
            t.q.load(qs + o);
            t.v = vs[b][j][col_s];
            t.beta = bs[b][j];
            return t;
        };
        float* dst = out + static_cast<size_t>(t0) * a.heads * a.vdim + static_cast<size_t>(h) * a.vdim + col;
        const size_t row_o = static_cast<size_t>(a.heads) * a.vdim;
        uint32_t j0 = 0;
        for (; j0 + 16 <= n; j0 += 16) {                     // sixteen tokens without a branch; lane i of a group stores token i
            float r[16];
            DeltaOperands<RQ> t = fetch(j0);
#pragma unroll
            for (uint32_t u = 0; u < 16; ++u) {
                const DeltaOperands<RQ> next = fetch(j0 + (u < 15 ? u + 1 : 15));
                r[u] = delta_token<RQ>(S, t);
                t = next;
            }
            const float x = group_transpose_sum(r, lg);
            if (live) dst[(j0 + lg) * row_o] = x;
        }
        for (; j0 < n; ++j0) {
            const float r = group_sum(delta_token<RQ>(S, fetch(j0)));
            if (lg == 0 && live) dst[j0 * row_o] = r;
        }
        __syncthreads();
    }
    if (live) S.store(sp);
}

// convolution + SiLU of channel `ch` (0 .. 2 qk + heads vdim) for one token; before(j): the input j tokens back
template <typename Before>
__device__ __forceinline__ float conv_silu(const float* w, uint32_t taps, float now, Before before) {
    float s = now * w[taps - 1];
    for (uint32_t j = 1; j < taps; ++j) s = fmaf(before(j), w[taps - 1 - j], s);
    return siluf(s);
}
__device__ __forceinline__ float decay_of(float a_log, float x) { return expf(-expf(a_log) * softplusf(x)); }
__device__ __forceinline__ float low_rank_dot(const void* w, size_t row, uint32_t ld, const float* x) {
    const __nv_bfloat16* r = static_cast<const __nv_bfloat16*>(w) + row * ld;
    float s = 0.f;
    for (uint32_t c = 0; c < ld; c += 8) {
        float f[8];
        load8(r + c, f);
#pragma unroll
        for (int i = 0; i < 8; ++i) s = fmaf(f[i], x[c + i], s);
    }
    return s;
}

// One token from the raw projection row: convolution, SiLU, unit norms, decays, gate and the state update.
template <int RQ>
__global__ void __launch_bounds__(SC_THREADS) delta_step_kernel(const __grid_constant__ hf2q_delta a, float* __restrict__ out, float* __restrict__ gate) {
    constexpr uint32_t DP = 32 * RQ;
    __shared__ __align__(16) float ks[DP], qs[DP], gs[DP], vs[SC_COLS];
    __shared__ float red[64];
    extern __shared__ __align__(16) float lr[];                     // a1 [a_rank_ld], g1 [g_rank_ld]
    pdl_trigger();
    const uint32_t h = blockIdx.x, slice = blockIdx.y, rep = a.heads / a.kv_heads, kvh = h / rep;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lg = lane & 15;
    const uint32_t col_s = warp * 2 + (lane >> 4), col0 = slice * SC_COLS, col = col0 + col_s;
    const uint32_t n_cols = min(static_cast<uint32_t>(SC_COLS), a.vdim - col0);
    const bool live = col < a.vdim;
    for (uint32_t i = threadIdx.x; i < a.dim; i += SC_THREADS)       // weights: towards L2 before the wait
        for (uint32_t c = 0; c < a.a_rank_ld; c += 64) prefetch_l2(static_cast<const __nv_bfloat16*>(a.a2) + (static_cast<size_t>(h) * a.dim + i) * a.a_rank_ld + c);
    pdl_wait();
    Vec<RQ> S;
    float* sp = a.s + (static_cast<size_t>(h) * a.vdim + (live ? col : 0)) * DP + 2 * lg;
    if (live) S.load(sp); else S.zero();
    const uint32_t pos = *a.pos, qk = a.kv_heads * a.dim;
    for (uint32_t i = threadIdx.x; i < a.a_rank_ld; i += SC_THREADS) lr[i] = a.proj[a.a1_off + i];
    for (uint32_t i = threadIdx.x; i < a.g_rank_ld; i += SC_THREADS) lr[a.a_rank_ld + i] = a.proj[a.g1_off + i];
    // the state ring has one column more than the taps look back, so this token's column is read by nobody
    auto channel = [&](uint32_t ch, const float* w, float now, bool keep) {
        float* st = a.conv_state + static_cast<size_t>(ch) * a.taps;
        const float v = conv_silu(w, a.taps, now, [&](uint32_t j) { return st[(pos + a.taps - j) % a.taps]; });
        if (keep) st[pos % a.taps] = now;
        return v;
    };
    float ss[2] = {0.f, 0.f};
    for (uint32_t i = threadIdx.x; i < DP; i += SC_THREADS) {
        float q = 0.f, k = 0.f;
        if (i < a.dim) {
            const uint32_t c = kvh * a.dim + i;
            const bool keep = slice == 0 && h % rep == 0;
            q = channel(c, a.q_conv + static_cast<size_t>(c) * a.taps, a.proj[a.q_off + c], keep);
            k = channel(qk + c, a.k_conv + static_cast<size_t>(c) * a.taps, a.proj[a.k_off + c], keep);
        }
        qs[i] = q;
        ks[i] = k;
        ss[0] += q * q;
        ss[1] += k * k;
    }
    if (threadIdx.x < SC_COLS) {
        float v = 0.f;
        if (threadIdx.x < n_cols) {
            const uint32_t c = h * a.vdim + col0 + threadIdx.x;
            v = channel(2 * qk + c, a.v_conv + static_cast<size_t>(c) * a.taps, a.proj[a.v_off + c], true);
        }
        vs[threadIdx.x] = v;
    }
    block_sum(ss, red);                                             // (its barrier also publishes lr and vs)
    const float iq = 1.0f / sqrtf(ss[0] + 1e-6f) / sqrtf(static_cast<float>(a.dim)), ik = 1.0f / sqrtf(ss[1] + 1e-6f);
    for (uint32_t i = threadIdx.x; i < DP; i += SC_THREADS) {
        qs[i] *= iq;
        ks[i] *= ik;
        gs[i] = i < a.dim ? decay_of(a.a_log[h], low_rank_dot(a.a2, static_cast<size_t>(h) * a.dim + i, a.a_rank_ld, lr) + a.dt_bias[h * a.dim + i]) : 0.f;
    }
    if (threadIdx.x < n_cols) {
        const uint32_t c = h * a.vdim + col0 + threadIdx.x;
        gate[c] = low_rank_dot(a.g2, c, a.g_rank_ld, lr + a.a_rank_ld);
    }
    __syncthreads();
    DeltaOperands<RQ> t;
    t.g.load(gs + 2 * lg);
    t.k.load(ks + 2 * lg);
    t.q.load(qs + 2 * lg);
    t.v = vs[col_s];
    t.beta = sigmoidf(a.proj[a.b_off + h]);
    const float r = group_sum(delta_token<RQ>(S, t));
    if (live) {
        S.store(sp);
        if (lg == 0) out[h * a.vdim + col] = r;
    }
}

// One CTA per token: a warp takes one head of q or k (or a head of v) at a time.
template <typename LR>
__global__ void __launch_bounds__(256) delta_prep_kernel(const __grid_constant__ hf2q_delta a, float* __restrict__ qkv, float* __restrict__ beta,
                                                         LR* __restrict__ a1, LR* __restrict__ g1) {
    pdl_trigger();
    pdl_wait();
    const uint32_t t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t pos = *a.pos, qk = a.kv_heads * a.dim;
    const float* row = a.proj + static_cast<size_t>(t) * a.ld;
    float* dst = qkv + static_cast<size_t>(t) * (2 * qk + a.heads * a.vdim);
    auto channel = [&](uint32_t ch, const float* w, uint32_t off) {
        return conv_silu(w, a.taps, row[off], [&](uint32_t j) {
            return j <= t ? row[static_cast<ptrdiff_t>(off) - static_cast<ptrdiff_t>(j) * a.ld]
                          : a.conv_state[static_cast<size_t>(ch) * a.taps + (pos + t + a.taps - j) % a.taps];
        });
    };
    for (uint32_t hd = warp; hd < 2 * a.kv_heads; hd += 8) {
        const bool is_k = hd >= a.kv_heads;
        const uint32_t c0 = (is_k ? hd - a.kv_heads : hd) * a.dim;
        const float* w = is_k ? a.k_conv : a.q_conv;
        float v[8], s = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const uint32_t i = lane + 32 * j;
            v[j] = i < a.dim ? channel((is_k ? qk : 0u) + c0 + i, w + static_cast<size_t>(c0 + i) * a.taps, (is_k ? a.k_off : a.q_off) + c0 + i) : 0.f;
            s += v[j] * v[j];
        }
        float inv = 1.0f / sqrtf(warp_sum(s) + 1e-6f);
        if (!is_k) inv /= sqrtf(static_cast<float>(a.dim));
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (lane + 32 * j < a.dim) dst[(is_k ? qk : 0u) + c0 + lane + 32 * j] = v[j] * inv;
    }
    for (uint32_t c = threadIdx.x; c < a.heads * a.vdim; c += 256)
        dst[2 * qk + c] = channel(2 * qk + c, a.v_conv + static_cast<size_t>(c) * a.taps, a.v_off + c);
    for (uint32_t h = threadIdx.x; h < a.heads; h += 256) beta[static_cast<size_t>(t) * a.heads + h] = sigmoidf(row[a.b_off + h]);
    for (uint32_t c = threadIdx.x; c < a.a_rank_ld; c += 256) a1[static_cast<size_t>(t) * a.a_rank_ld + c] = from_f32<LR>(row[a.a1_off + c]);
    for (uint32_t c = threadIdx.x; c < a.g_rank_ld; c += 256) g1[static_cast<size_t>(t) * a.g_rank_ld + c] = from_f32<LR>(row[a.g1_off + c]);
}

__global__ void __launch_bounds__(256) delta_decay_kernel(const float* __restrict__ a_log, const float* __restrict__ dt_bias, uint32_t dim, uint32_t per_token,
                                                          uint64_t n, float* __restrict__ g) {
    pdl_trigger();
    pdl_wait();
    const uint64_t stride = static_cast<uint64_t>(gridDim.x) * blockDim.x;
    for (uint64_t i = static_cast<uint64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < n; i += stride) {
        const uint32_t c = static_cast<uint32_t>(i % per_token);
        g[i] = decay_of(a_log[c / dim], g[i] + dt_bias[c]);
    }
}

// ---------------------------------------------------------------- state space with a scalar decay
__device__ __forceinline__ uint32_t ssd_channels(const hf2q_ssd& a) { return a.heads * a.vdim + 2 * a.groups * a.state; }

// S <- keep S + dt B x^T;  y = S^T C + d x
template <int RQ>
__global__ void __launch_bounds__(SC_THREADS) ssd_scan_kernel(const __grid_constant__ hf2q_ssd a, uint32_t m, const float* __restrict__ xbc,
                                                              const float* __restrict__ dt, const float* __restrict__ la, float* __restrict__ y) {
    constexpr uint32_t DP = 32 * RQ;
    extern __shared__ __align__(16) float dsm[];                    // B, C: [2][SC_TB][DP] each
    float* ks = dsm;
    float* qs = dsm + 2 * SC_TB * DP;
    __shared__ __align__(16) float vs[2][SC_TB][SC_COLS];
    __shared__ float gk[2][SC_TB], gw[2][SC_TB];                    // decay, step size
    pdl_trigger();
    pdl_wait();
    const uint32_t h = blockIdx.x, slice = blockIdx.y, grp = h / (a.heads / a.groups);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lg = lane & 15;
    const uint32_t col_s = warp * 2 + (lane >> 4), col0 = slice * SC_COLS, col = col0 + col_s;
    const uint32_t n_cols = min(static_cast<uint32_t>(SC_COLS), a.vdim - col0);
    const bool live = col < a.vdim;
    const uint32_t channels = ssd_channels(a), inner = a.heads * a.vdim;
    // the convolution's reader has finished: the last inputs go to the state
    for (uint32_t i = (blockIdx.y * gridDim.x + blockIdx.x) * SC_THREADS + threadIdx.x; i < channels; i += gridDim.x * gridDim.y * SC_THREADS) {
        const uint32_t pos = *a.pos, keep = min(a.taps - 1, m);
        for (uint32_t j = 0; j < keep; ++j)
            a.conv_state[static_cast<size_t>(i) * a.taps + (pos + m - 1 - j) % a.taps] = a.proj[static_cast<size_t>(m - 1 - j) * a.ld + a.off + i];
    }
    for (uint32_t i = threadIdx.x; i < 4 * SC_TB * DP; i += SC_THREADS) dsm[i] = 0.f;
    for (uint32_t i = threadIdx.x; i < 2 * SC_TB * SC_COLS; i += SC_THREADS) (&vs[0][0][0])[i] = 0.f;
    __syncthreads();
    auto stage = [&](uint32_t t0, uint32_t b) {
        const uint32_t n = min(static_cast<uint32_t>(SC_TB), m - t0);
        const float* row = xbc + static_cast<size_t>(t0) * channels;
        stage_rows(ks + b * SC_TB * DP, DP, row + inner + grp * a.state, channels, n, a.state);
        stage_rows(qs + b * SC_TB * DP, DP, row + inner + (a.groups + grp) * a.state, channels, n, a.state);
        stage_rows(vs[b][0], SC_COLS, row + h * a.vdim + col0, channels, n, n_cols);
        if (threadIdx.x < n) {
            const size_t o = static_cast<size_t>(t0 + threadIdx.x) * a.heads + h;
            gk[b][threadIdx.x] = expf(la[o]);
            gw[b][threadIdx.x] = dt[o];
        }
        cp_async_commit();
    };
    Vec<RQ> S;
    float* sp = a.s + (static_cast<size_t>(h) * a.vdim + (live ? col : 0)) * DP + 2 * lg;
    const float skip = a.d[h];
    if (live) S.load(sp); else S.zero();
    stage(0, 0);
    for (uint32_t t0 = 0, b = 0; t0 < m; t0 += SC_TB, b ^= 1) {
        if (t0 + SC_TB < m) { stage(t0 + SC_TB, b ^ 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        const uint32_t n = min(static_cast<uint32_t>(SC_TB), m - t0);
        struct Operands { Vec<RQ> k, q; float keep, write, v; };
        auto fetch = [&](uint32_t j) {
            Operands t;
            t.k.load(ks + (b * SC_TB + j) * DP + 2 * lg);
            t.q.load(qs + (b * SC_TB + j) * DP + 2 * lg);
            t.keep = gk[b][j];
            t.write = gw[b][j];
            t.v = vs[b][j][col_s];
            return t;
        };
        auto finish = [&](uint32_t j, float s) {
            if (live) y[static_cast<size_t>(t0 + j) * inner + static_cast<size_t>(h) * a.vdim + col] = s + skip * vs[b][j][col_s];
        };
        uint32_t j0 = 0;
        for (; j0 + 16 <= n; j0 += 16) {                     // sixteen tokens without a branch; lane i of a group finishes token i
            float r[16];
            Operands t = fetch(j0);
#pragma unroll
            for (uint32_t u = 0; u < 16; ++u) {
                const Operands next = fetch(j0 + (u < 15 ? u + 1 : 15));
                S.decay_axpy(t.keep, t.k, t.write * t.v);
                r[u] = S.dot(t.q);
                t = next;
            }
            finish(j0 + lg, group_transpose_sum(r, lg));
        }
        for (; j0 < n; ++j0) {
            const Operands t = fetch(j0);
            S.decay_axpy(t.keep, t.k, t.write * t.v);
            const float r = group_sum(S.dot(t.q));
            if (lg == 0) finish(j0, r);
        }
        __syncthreads();
    }
    if (live) S.store(sp);
}

__device__ __forceinline__ void ssd_gates(const hf2q_ssd& a, uint32_t h, float raw, float& dt, float& la) {
    dt = softplusf(raw + a.dt_bias[h]);
    la = -expf(a.a_log[h]) * dt;
}
template <typename Before>
__device__ __forceinline__ float conv_bias_silu(const float* w, float bias, uint32_t taps, float now, Before before) {
    float s = fmaf(now, w[taps - 1], bias);
    for (uint32_t j = 1; j < taps; ++j) s = fmaf(before(j), w[taps - 1 - j], s);
    return siluf(s);
}

// One CTA per token.
__global__ void __launch_bounds__(256) ssd_prep_kernel(const __grid_constant__ hf2q_ssd a, float* __restrict__ xbc, float* __restrict__ dt, float* __restrict__ la) {
    pdl_trigger();
    pdl_wait();
    const uint32_t t = blockIdx.x, pos = *a.pos, channels = ssd_channels(a);
    const float* row = a.proj + static_cast<size_t>(t) * a.ld + a.off;
    float* dst = xbc + static_cast<size_t>(t) * channels;
    for (uint32_t c = threadIdx.x; c < channels; c += 256)
        dst[c] = conv_bias_silu(a.conv + static_cast<size_t>(c) * a.taps, a.conv_bias[c], a.taps, row[c], [&](uint32_t j) {
            return j <= t ? row[static_cast<ptrdiff_t>(c) - static_cast<ptrdiff_t>(j) * a.ld] : a.conv_state[static_cast<size_t>(c) * a.taps + (pos + t + a.taps - j) % a.taps];
        });
    for (uint32_t h = threadIdx.x; h < a.heads; h += 256) {
        const size_t o = static_cast<size_t>(t) * a.heads + h;
        ssd_gates(a, h, row[channels + h], dt[o], la[o]);
    }
}

// One token from the raw projection row: convolution, SiLU, step size and the state update.
template <int RQ>
__global__ void __launch_bounds__(SC_THREADS) ssd_step_kernel(const __grid_constant__ hf2q_ssd a, float* __restrict__ y) {
    constexpr uint32_t DP = 32 * RQ;
    __shared__ __align__(16) float ks[DP], qs[DP], vs[SC_COLS];
    pdl_trigger();
    const uint32_t h = blockIdx.x, slice = blockIdx.y, rep = a.heads / a.groups, grp = h / rep;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lg = lane & 15;
    const uint32_t col_s = warp * 2 + (lane >> 4), col0 = slice * SC_COLS, col = col0 + col_s;
    const uint32_t n_cols = min(static_cast<uint32_t>(SC_COLS), a.vdim - col0);
    const bool live = col < a.vdim;
    pdl_wait();
    Vec<RQ> S;
    float* sp = a.s + (static_cast<size_t>(h) * a.vdim + (live ? col : 0)) * DP + 2 * lg;
    if (live) S.load(sp); else S.zero();
    const uint32_t pos = *a.pos, channels = ssd_channels(a), inner = a.heads * a.vdim;
    const float* row = a.proj + a.off;
    // the state ring has one column more than the taps look back, so this token's column is read by nobody
    auto channel = [&](uint32_t c, bool keep) {
        float* st = a.conv_state + static_cast<size_t>(c) * a.taps;
        const float now = row[c];
        const float v = conv_bias_silu(a.conv + static_cast<size_t>(c) * a.taps, a.conv_bias[c], a.taps, now, [&](uint32_t j) { return st[(pos + a.taps - j) % a.taps]; });
        if (keep) st[pos % a.taps] = now;
        return v;
    };
    const bool first = slice == 0 && h % rep == 0;
    for (uint32_t i = threadIdx.x; i < 2 * DP; i += SC_THREADS) {
        const uint32_t j = i % DP;
        const float v = j < a.state ? channel(inner + (i < DP ? grp : a.groups + grp) * a.state + j, first) : 0.f;
        (i < DP ? ks : qs)[j] = v;
    }
    if (threadIdx.x < SC_COLS) vs[threadIdx.x] = threadIdx.x < n_cols ? channel(h * a.vdim + col0 + threadIdx.x, true) : 0.f;
    float dt, la;
    ssd_gates(a, h, row[channels + h], dt, la);
    __syncthreads();
    Vec<RQ> k, q;
    k.load(ks + 2 * lg);
    q.load(qs + 2 * lg);
    S.decay_axpy(expf(la), k, dt * vs[col_s]);
    const float r = group_sum(S.dot(q));
    if (live) {
        S.store(sp);
        if (lg == 0) y[h * a.vdim + col] = r + a.d[h] * vs[col_s];
    }
}

bool ssd_ok(const hf2q_ssd* a) {
    return a && a->proj && a->conv && a->conv_bias && a->dt_bias && a->a_log && a->d && a->conv_state && a->s && a->pos && a->heads && a->groups &&
           a->heads % a->groups == 0 && a->state && a->state <= 256 && a->vdim && a->taps;
}
template <int RQ>
cudaError_t launch_ssd_scan(const hf2q_ssd& a, uint32_t m, const float* xbc, const float* dt, const float* la, float* y, cudaStream_t st) {
    static PerDeviceFlag flag;
    const size_t smem = 4ull * SC_TB * 32 * RQ * sizeof(float);
    if (const cudaError_t e = ensure_max_dynamic_smem(ssd_scan_kernel<RQ>, static_cast<int>(smem), flag); e != cudaSuccess) return e;
    return launch_pdl(ssd_scan_kernel<RQ>, dim3(a.heads, (a.vdim + SC_COLS - 1) / SC_COLS), dim3(SC_THREADS), smem, st, a, m, xbc, dt, la, y);
}

bool delta_ok(const hf2q_delta* a) {
    return a && a->proj && a->q_conv && a->k_conv && a->v_conv && a->a_log && a->dt_bias && a->a2 && a->g2 && a->conv_state && a->s && a->pos &&
           a->heads && a->kv_heads && a->heads % a->kv_heads == 0 && a->dim && a->dim <= 256 && a->vdim && a->taps && a->a_rank_ld % 8 == 0 &&
           a->g_rank_ld % 8 == 0 && a->a_rank_ld && a->g_rank_ld;
}
template <int RQ>
cudaError_t launch_scan(const hf2q_delta& a, uint32_t m, const float* qkv, const float* beta, const float* g, float* out, cudaStream_t st) {
    static PerDeviceFlag flag;
    const size_t smem = 6ull * SC_TB * 32 * RQ * sizeof(float);
    if (const cudaError_t e = ensure_max_dynamic_smem(delta_scan_kernel<RQ>, static_cast<int>(smem), flag); e != cudaSuccess) return e;
    return launch_pdl(delta_scan_kernel<RQ>, dim3(a.heads, (a.vdim + SC_COLS - 1) / SC_COLS), dim3(SC_THREADS), smem, st, a, m, qkv, beta, g, out);
}

template <int RQ>
cudaError_t launch_mlstm(const hf2q_mlstm& a, uint32_t m, float* out, cudaStream_t st) {
    static PerDeviceFlag flag;
    const size_t smem = 4ull * SC_TB * 32 * RQ * sizeof(float);
    if (const cudaError_t e = ensure_max_dynamic_smem(mlstm_kernel<RQ>, static_cast<int>(smem), flag); e != cudaSuccess) return e;
    return launch_pdl(mlstm_kernel<RQ>, dim3(a.heads, (a.vdim + SC_COLS - 1) / SC_COLS), dim3(SC_THREADS), smem, st, a, m, out);
}

#define HF2Q_RQ_CASES(F) F(1) F(2) F(3) F(4) F(5) F(6) F(7) F(8)

}  // namespace
}  // namespace hf2q

using namespace hf2q;
using namespace hf2q::seq;

extern "C" {

HF2Q_API int32_t hf2q_cuda_mlstm(hf2q_ctx* ctx, void* stream, const hf2q_mlstm* a, uint32_t m, float* out) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!a || !a->proj || !a->i_bias || !a->f_bias || !a->s || !a->n || !a->mx || !out || a->heads == 0 || a->dim == 0 || a->vdim == 0 || a->dim > 256 ||
        !(a->gate_cap > 0.f))
        return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "mlstm: null pointer, or a size outside dim 1..256");
    if (m == 0) return HF2Q_OK;
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    cudaError_t e = cudaErrorInvalidValue;
    switch ((a->dim + 31) / 32) {
#define F(RQ) case RQ: e = launch_mlstm<RQ>(*a, m, out, st); break;
        HF2Q_RQ_CASES(F)
#undef F
        default: break;
    }
    return ctx_cuda_result(ctx, e, "mlstm", 1);
}

HF2Q_API int32_t hf2q_cuda_delta_step(hf2q_ctx* ctx, void* stream, const hf2q_delta* a, float* out, float* gate) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!delta_ok(a) || !out || !gate) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "delta_step: null pointer or an unsupported size");
    const dim3 grid(a->heads, (a->vdim + SC_COLS - 1) / SC_COLS);
    const size_t smem = static_cast<size_t>(a->a_rank_ld + a->g_rank_ld) * 4;
    if (smem > 32 * 1024) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "delta_step: rank too large");
    cudaError_t e = cudaErrorInvalidValue;
    switch ((a->dim + 31) / 32) {
#define F(RQ) case RQ: e = launch_pdl(delta_step_kernel<RQ>, grid, dim3(SC_THREADS), smem, static_cast<cudaStream_t>(stream), *a, out, gate); break;
        HF2Q_RQ_CASES(F)
#undef F
        default: break;
    }
    return ctx_cuda_result(ctx, e, "delta_step", 1);
}

HF2Q_API int32_t hf2q_cuda_delta_prep(hf2q_ctx* ctx, void* stream, const hf2q_delta* a, uint32_t m, float* qkv, float* beta, void* a1, void* g1,
                                      uint32_t lr_dtype) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!delta_ok(a) || !qkv || !beta || !a1 || !g1) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "delta_prep: null pointer or an unsupported size");
    if (m == 0) return HF2Q_OK;
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    cudaError_t e = cudaErrorInvalidValue;
    if (lr_dtype == HF2Q_DT_F32)
        e = launch_pdl(delta_prep_kernel<float>, dim3(m), dim3(256), 0, st, *a, qkv, beta, static_cast<float*>(a1), static_cast<float*>(g1));
    else if (lr_dtype == HF2Q_DT_BF16)
        e = launch_pdl(delta_prep_kernel<__nv_bfloat16>, dim3(m), dim3(256), 0, st, *a, qkv, beta, static_cast<__nv_bfloat16*>(a1), static_cast<__nv_bfloat16*>(g1));
    return ctx_cuda_result(ctx, e, "delta_prep", 1);
}

HF2Q_API int32_t hf2q_cuda_delta_decay(hf2q_ctx* ctx, void* stream, const hf2q_delta* a, uint32_t m, float* g) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!delta_ok(a) || !g) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "delta_decay: null pointer or an unsupported size");
    if (m == 0) return HF2Q_OK;
    const uint64_t n = static_cast<uint64_t>(m) * a->heads * a->dim, want = (n + 255) / 256, cap = static_cast<uint64_t>(ctx_sm_count(ctx)) * 16;
    const cudaError_t e = launch_pdl(delta_decay_kernel, dim3(static_cast<unsigned>(want < cap ? want : cap)), dim3(256), 0, static_cast<cudaStream_t>(stream),
                                     a->a_log, a->dt_bias, a->dim, a->heads * a->dim, n, g);
    return ctx_cuda_result(ctx, e, "delta_decay", 1);
}

HF2Q_API int32_t hf2q_cuda_delta_scan(hf2q_ctx* ctx, void* stream, const hf2q_delta* a, uint32_t m, const float* qkv, const float* beta, const float* g,
                                      float* out) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!delta_ok(a) || !qkv || !beta || !g || !out) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "delta_scan: null pointer or an unsupported size");
    if (m == 0) return HF2Q_OK;
    const cudaStream_t st = static_cast<cudaStream_t>(stream);
    cudaError_t e = cudaErrorInvalidValue;
    switch ((a->dim + 31) / 32) {
#define F(RQ) case RQ: e = launch_scan<RQ>(*a, m, qkv, beta, g, out, st); break;
        HF2Q_RQ_CASES(F)
#undef F
        default: break;
    }
    return ctx_cuda_result(ctx, e, "delta_scan", 1);
}

HF2Q_API int32_t hf2q_cuda_ssd_step(hf2q_ctx* ctx, void* stream, const hf2q_ssd* a, float* y) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!ssd_ok(a) || !y) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "ssd_step: null pointer or an unsupported size");
    const dim3 grid(a->heads, (a->vdim + SC_COLS - 1) / SC_COLS);
    cudaError_t e = cudaErrorInvalidValue;
    switch ((a->state + 31) / 32) {
#define F(RQ) case RQ: e = launch_pdl(ssd_step_kernel<RQ>, grid, dim3(SC_THREADS), 0, static_cast<cudaStream_t>(stream), *a, y); break;
        HF2Q_RQ_CASES(F)
#undef F
        default: break;
    }
    return ctx_cuda_result(ctx, e, "ssd_step", 1);
}

HF2Q_API int32_t hf2q_cuda_ssd_prep(hf2q_ctx* ctx, void* stream, const hf2q_ssd* a, uint32_t m, float* xbc, float* dt, float* la) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!ssd_ok(a) || !xbc || !dt || !la) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "ssd_prep: null pointer or an unsupported size");
    if (m == 0) return HF2Q_OK;
    return ctx_cuda_result(ctx, launch_pdl(ssd_prep_kernel, dim3(m), dim3(256), 0, static_cast<cudaStream_t>(stream), *a, xbc, dt, la), "ssd_prep", 1);
}

HF2Q_API int32_t hf2q_cuda_ssd_scan(hf2q_ctx* ctx, void* stream, const hf2q_ssd* a, uint32_t m, const float* xbc, const float* dt, const float* la, float* y) {
    if (!ctx) return HF2Q_ERR_INVALID_ARGUMENT;
    if (!ssd_ok(a) || !xbc || !dt || !la || !y) return ctx_fail(ctx, HF2Q_ERR_INVALID_ARGUMENT, "ssd_scan: null pointer or an unsupported size");
    if (m == 0) return HF2Q_OK;
    cudaError_t e = cudaErrorInvalidValue;
    switch ((a->state + 31) / 32) {
#define F(RQ) case RQ: e = launch_ssd_scan<RQ>(*a, m, xbc, dt, la, y, static_cast<cudaStream_t>(stream)); break;
        HF2Q_RQ_CASES(F)
#undef F
        default: break;
    }
    return ctx_cuda_result(ctx, e, "ssd_scan", 1);
}

}  // extern "C"
