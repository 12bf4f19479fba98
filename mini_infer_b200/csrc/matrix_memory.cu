// Matrix memories with one gate per head: a request keeps, per head, a matrix S [d, dv] (float) and
//
//   S_t = keep_t S_(t-1) + write_t k_t v_t^T          o_t = S_t^T q_t
//
// Two sources of the gates:
//
//   fixed decay     keep_t = decay[h], write_t = 1 (linear attention with a constant decay per head)
//   log gates       a log input gate i and a log forget gate f per token and head, and a running maximum m that keeps
//                   the exponentials bounded:  m_t = max(f + m_(t-1), i),  keep = exp(f + m_(t-1) - m_t),
//                   write = exp(i - m_t).  The sum of the keys, n_t = keep n_(t-1) + write k_t, is one more column of S
//                   (a value that is always 1); the read-out is divided by max(|n_t . q_t|, exp(-m_t)) + 1e-6.
//
// Forms of the same recurrence:
//
//   memory_gates    the log gates of a step's tokens and the chain of m (one block per request and head)
//   memory_walk     token by token, a block per (request, head, 16 value columns): the order of a token's additions
//                   depends on the model's sizes only, whatever the cut of the step
//   memory_chunks   long portions on the tensor cores, 64 tokens at a time (bfloat16 path): see below
//   memory_decode   one token per request: gates, state, read-out, output norm and output gate in one launch
//   memory_finish   division, RMS norm per head, weight, logistic gate
//
// q, k and v are columns of one row of float projections; `act` 1 puts them through silu first.  State of a slot:
// S [H][d][dv] at `s_off`, and with log gates n [H][d] at `n_off` and m [H] at `m_off`.

#include <cooperative_groups.h>

#include "common.cuh"

namespace cg = cooperative_groups;

namespace mi {
namespace mem {

__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
// log(logistic(x)) = -log(1 + e^-x), without overflow on either side
__device__ __forceinline__ float log_sigmoid_f(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ void copy_async_f32(float* smem_dst, const float* src) {
    const uint32_t dst = static_cast<uint32_t>(__cvta_generic_to_shared(smem_dst));
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(dst), "l"(src));
}
__device__ __forceinline__ void copy_async_16(float* smem_dst, const float* src) {
    const uint32_t dst = static_cast<uint32_t>(__cvta_generic_to_shared(smem_dst));
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(src));
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
__device__ __forceinline__ void copy_async_wait_but_one() { asm volatile("cp.async.wait_group 1;\n" ::: "memory"); }

// Columns of a projection row, and what is done to them.
struct Rows {
    const float* p;         // [T, ld]
    int64_t ld;
    int q, k, v;            // first columns of q, k (H x d each) and v (H x dv)
    int act;                // 1: silu
    float q_scale;
};

// The state of a request: float row `slot` of `base`.
struct State {
    float* base;
    int64_t stride;
    int64_t s_off, n_off, m_off;
    __device__ __forceinline__ float* row(int slot) const { return base + (int64_t)slot * stride; }
};

// What a token of one head brings besides its vectors: keep, write, exp(-m) and f; and i, m, m before it, 0.
struct LogGates {
    const float* p;         // [T, ld] projections
    int64_t ld;
    int i, f;               // first columns of the H input gates and of the H forget gates
    const float* bi;        // [H] biases
    const float* bf;
    float cap;              // gate = cap tanh(gate / cap)
};
__device__ __forceinline__ void log_gates(const LogGates& g, int64_t t, int h, float& li, float& lf) {
    const float* row = g.p + t * g.ld;
    li = g.cap * tanhf((row[g.i + h] + g.bi[h]) / g.cap);
    lf = log_sigmoid_f(g.cap * tanhf((row[g.f + h] + g.bf[h]) / g.cap));
}

// One block per (head, request).  The gates of 256 tokens are formed side by side, one thread runs the chain of m over
// them (an addition and a maximum per token), and the exponentials are formed side by side again.
// gates [T][H] = (keep, write, exp(-m), f);  logs [T][H] = (i, m, m before, 0) or null.
// SCAN: the step m -> max(f + m, i) as the pair (f, i), pairs composed by warps and then over the warps: the sums of f
// run in another order than in the chain, which is what the chunks of long portions do with them anyway.
template <bool SCAN>
__global__ void __launch_bounds__(256)
memory_gates_kernel(LogGates lg, State st, const int* __restrict__ q_start, const int* __restrict__ state_slot,
                    float4* __restrict__ gates, float4* __restrict__ logs, int H) {
    __shared__ float si[256], sf[256], sm[257], wf[8], wi[8];
    wait_for_earlier_kernels();
    const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
    const int q0 = q_start[b], n = q_start[b + 1] - q0;
    float* m_state = st.row(state_slot[b]) + st.m_off + h;
    if (tid == 0) sm[0] = *m_state;
    for (int c0 = 0; c0 < n; c0 += 256) {
        const int nc = min(256, n - c0);
        float li = -INFINITY, lf = 0.f;                  // (beyond the portion: a step that changes nothing)
        if (tid < nc) log_gates(lg, q0 + c0 + tid, h, li, lf);
        if (SCAN) {
            const int lane = tid & 31, warp = tid >> 5;
            float cf = lf, ci = li;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float pf = __shfl_up_sync(0xffffffffu, cf, o), pi = __shfl_up_sync(0xffffffffu, ci, o);
                if (lane >= o) { ci = fmaxf(cf + pi, ci); cf += pf; }
            }
            if (lane == 31) { wf[warp] = cf; wi[warp] = ci; }
            __syncthreads();
            float m = sm[0];
            for (int w = 0; w < warp; ++w) m = fmaxf(wf[w] + m, wi[w]);
            const float mine = fmaxf(cf + m, ci);
            __syncthreads();                             // sm[0] has been read
            sm[tid + 1] = mine;
            __syncthreads();
        } else {
        si[tid] = li;
        sf[tid] = lf;
        __syncthreads();
        if (tid == 0) {
            // eight tokens' gates are asked for before the first of them: the chain is an addition and a maximum
            float m = sm[0];
            for (int t = 0; t < 256; t += 8) {
                float f8[8], i8[8];
#pragma unroll
                for (int k = 0; k < 8; ++k) { f8[k] = sf[t + k]; i8[k] = si[t + k]; }
#pragma unroll
                for (int k = 0; k < 8; ++k) { m = fmaxf(f8[k] + m, i8[k]); f8[k] = m; }
#pragma unroll
                for (int k = 0; k < 8; ++k) sm[t + k + 1] = f8[k];
                if (t + 8 >= nc) break;
            }
        }
        __syncthreads();
        }
        if (tid < nc) {
            const float before = sm[tid], m = sm[tid + 1];
            const int64_t at = (int64_t)(q0 + c0 + tid) * H + h;
            gates[at] = make_float4(expf(lf + before - m), expf(li - m), expf(-m), lf);
            if (logs) logs[at] = make_float4(li, m, before, 0.f);
        }
        __syncthreads();
        if (tid == 0) sm[0] = sm[nc];
    }
    if (tid == 0 && n > 0) *m_state = sm[0];
}

// ---------------------------------------------------------------------------
// The walk.  Block = 128 threads = 16 value columns x 8 lanes; lane r of a column holds, of that column of S, the rows
// 4 (r + 8 m) .. + 3.  Tokens come 16 at a time, the next 16 on their way (cp.async) while these are walked; the
// read-outs of four tokens are summed over the lanes together.  With log gates column dv is n (its value is 1).
// ---------------------------------------------------------------------------
constexpr int kLanes = 8, kCols = 16, kChunk = 16;

template <int RP, bool LOG>
__global__ void __launch_bounds__(128)
memory_walk_kernel(Rows in, State st, const float4* __restrict__ gates, const float* __restrict__ decay,
                   const int* __restrict__ q_start, const int* __restrict__ state_slot, float* __restrict__ out,
                   float* __restrict__ den, int H, int d, int dv, int vec) {
    extern __shared__ __align__(16) float sm[];
    constexpr int DP = RP * kLanes, MV = RP / 4;
    constexpr int kBuf = kChunk * (2 * DP + kCols + 4);
    float* os = sm + 2 * kBuf;                          // [16][16] results
    wait_for_earlier_kernels();
    const int b = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * kCols;
    const int tid = threadIdx.x, r = tid & (kLanes - 1), lc = tid / kLanes, col = col0 + lc;
    const bool is_n = LOG && col == dv;
    const int q0 = q_start[b], n = q_start[b + 1] - q0;
    float* row = st.row(state_slot[b]);
    float* S = row + st.s_off + (int64_t)h * d * dv;
    float* N = row + st.n_off + (int64_t)h * d;
    float s[RP];
#pragma unroll
    for (int m = 0; m < MV; ++m)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int i = 4 * (r + kLanes * m) + x;
            float v = 0.f;
            if (i < d) { if (col < dv) v = S[(int64_t)i * dv + col]; else if (is_n) v = N[i]; }
            s[4 * m + x] = v;
        }
    const float fixed = LOG ? 0.f : decay[h];
    // rows beyond the head's size are never copied to: zero them once in both buffers
    if (d < DP)
        for (int idx = tid; idx < 2 * 2 * kChunk * (DP - d); idx += 128) {
            const int i = d + idx % (DP - d), w = idx / (DP - d);
            sm[(w / (2 * kChunk)) * kBuf + (w % (2 * kChunk)) * DP + i] = 0.f;
        }
    const int n_cols = max(0, min(kCols, dv - col0));

    auto fetch = [&](int c0, float* buf) {
        const int nc = min(kChunk, n - c0);
        float* ks = buf + kChunk * DP;
        float* vs = ks + kChunk * DP;
        float* gs = vs + kChunk * kCols;
        const float* base = in.p + (int64_t)(q0 + c0) * in.ld;
        if (vec) {
            const int d4 = d / 4;
            for (int idx = tid; idx < nc * d4; idx += 128) {
                const int tt = idx / d4, i = 4 * (idx - tt * d4);
                copy_async_16(buf + tt * DP + i, base + tt * in.ld + in.q + h * d + i);
                copy_async_16(ks + tt * DP + i, base + tt * in.ld + in.k + h * d + i);
            }
        } else {
            for (int idx = tid; idx < nc * d; idx += 128) {
                const int tt = idx / d, i = idx - tt * d;
                copy_async_f32(buf + tt * DP + i, base + tt * in.ld + in.q + h * d + i);
                copy_async_f32(ks + tt * DP + i, base + tt * in.ld + in.k + h * d + i);
            }
        }
        for (int idx = tid; idx < nc * n_cols; idx += 128) {
            const int tt = idx / n_cols, c = idx - tt * n_cols;
            copy_async_f32(vs + tt * kCols + c, base + tt * in.ld + in.v + (int64_t)h * dv + col0 + c);
        }
        if (LOG && tid < nc)
            copy_async_16(gs + 4 * tid, reinterpret_cast<const float*>(gates + (int64_t)(q0 + c0 + tid) * H + h));
    };

    fetch(0, sm);
    copy_async_commit();
    int which = 0;
    for (int c0 = 0; c0 < n; c0 += kChunk, which ^= 1) {
        const int nc = min(kChunk, n - c0);
        float* qs = sm + which * kBuf;
        float* ks = qs + kChunk * DP;
        float* vs = ks + kChunk * DP;
        const float* gs = vs + kChunk * kCols;
        if (c0 + kChunk < n) fetch(c0 + kChunk, sm + (which ^ 1) * kBuf);
        copy_async_commit();
        copy_async_wait_but_one();
        __syncthreads();
        if (in.act) {
            for (int idx = tid; idx < nc * d; idx += 128) {
                const int tt = idx / d, i = idx - tt * d;
                qs[tt * DP + i] = silu_f(qs[tt * DP + i]);
                ks[tt * DP + i] = silu_f(ks[tt * DP + i]);
            }
            for (int idx = tid; idx < nc * n_cols; idx += 128) {
                const int tt = idx / n_cols, c = idx - tt * n_cols;
                vs[tt * kCols + c] = silu_f(vs[tt * kCols + c]);
            }
            __syncthreads();
        }
        for (int t4 = 0; t4 < nc; t4 += 4) {
            float o_part[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int u4 = 0; u4 < 4; ++u4) {
                const int tt = t4 + u4;
                if (tt < nc) {
                    const float4* kq = reinterpret_cast<const float4*>(ks + tt * DP);
                    const float4* qq = reinterpret_cast<const float4*>(qs + tt * DP);
                    const float keep = LOG ? gs[4 * tt] : fixed;
                    const float v = is_n ? 1.f : vs[tt * kCols + lc];
                    const float u = LOG ? gs[4 * tt + 1] * v : v;
                    float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
                    for (int m = 0; m < MV; ++m) {
                        const float4 k4 = kq[r + kLanes * m], q4 = qq[r + kLanes * m];
                        s[4 * m] = keep * s[4 * m] + k4.x * u; s[4 * m + 1] = keep * s[4 * m + 1] + k4.y * u;
                        s[4 * m + 2] = keep * s[4 * m + 2] + k4.z * u; s[4 * m + 3] = keep * s[4 * m + 3] + k4.w * u;
                        o0 += s[4 * m] * q4.x; o1 += s[4 * m + 1] * q4.y; o2 += s[4 * m + 2] * q4.z; o3 += s[4 * m + 3] * q4.w;
                    }
                    o_part[u4] = (o0 + o1) + (o2 + o3);
                }
            }
#pragma unroll
            for (int sh = 1; sh < kLanes; sh <<= 1)
#pragma unroll
                for (int u4 = 0; u4 < 4; ++u4) o_part[u4] += __shfl_xor_sync(0xffffffffu, o_part[u4], sh);
            if (r == 0) {
#pragma unroll
                for (int u4 = 0; u4 < 4; ++u4)
                    if (t4 + u4 < nc) os[(t4 + u4) * kCols + lc] = o_part[u4] * in.q_scale;
            }
        }
        __syncthreads();
        for (int idx = tid; idx < nc * kCols; idx += 128) {
            const int tt = idx / kCols, c = col0 + idx % kCols;
            const int64_t t = q0 + c0 + tt;
            if (c < dv) out[t * H * dv + (int64_t)h * dv + c] = os[idx];
            else if (LOG && c == dv) den[t * H + h] = os[idx];
        }
    }
#pragma unroll
    for (int m = 0; m < MV; ++m)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int i = 4 * (r + kLanes * m) + x;
            if (i < d) { if (col < dv) S[(int64_t)i * dv + col] = s[4 * m + x]; else if (is_n) N[i] = s[4 * m + x]; }
        }
}

// The same for groups of whole fours on 16-byte boundaries, kept in registers between the sum and the result: a warp per
// group of up to 512 columns (ONE_WARP; eight groups a block), a block of 256 threads per group of up to 8,192.
template <typename AT, typename GT, int VPT, bool ONE_WARP>
__global__ void __launch_bounds__(256)
memory_finish_vec_kernel(const float* __restrict__ o, const float* __restrict__ den, const float4* __restrict__ gates,
                         const GT* __restrict__ gate, int64_t ld_gate, const float* __restrict__ w, AT* __restrict__ out,
                         int n, int gs, float eps, int64_t total) {
    __shared__ float scratch[32];
    wait_for_earlier_kernels();
    const int groups = n / gs;
    const int64_t at = ONE_WARP ? (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5) : (int64_t)blockIdx.x;     // (token, group)
    if (at >= total) return;                                       // (one warp: whole warps leave, and no block-wide barrier follows)
    const int64_t t = at / groups;
    const int h = (int)(at - t * groups);
    constexpr int TH = ONE_WARP ? 32 : 256;
    const int i0 = ONE_WARP ? threadIdx.x & 31 : threadIdx.x, nv = gs / 4;
    const float4* row = reinterpret_cast<const float4*>(o + at * gs);
    const float4* wr = reinterpret_cast<const float4*>(w + h * gs);
    const GT* gr = gate + t * ld_gate + h * gs;
    AT* orow = out + at * gs;
    const float inv = den ? 1.0f / (fmaxf(fabsf(den[at]), gates[at].z) + 1e-6f) : 1.0f;
    float4 v[VPT];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int i = i0 + TH * j;
        v[j] = i < nv ? row[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        v[j].x *= inv; v[j].y *= inv; v[j].z *= inv; v[j].w *= inv;
        ss += (v[j].x * v[j].x + v[j].y * v[j].y) + (v[j].z * v[j].z + v[j].w * v[j].w);
    }
    ss = ONE_WARP ? warp_sum(ss) : block_sum(ss, scratch);
    const float rr = 1.0f / sqrtf(ss / (float)gs + eps);
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int i = i0 + TH * j, c = 4 * i;
        if (i < nv) {
            const float4 u = wr[i];
            store4(orow + c, make_float4(v[j].x * rr * u.x * sigmoid_f(to_float(gr[c])), v[j].y * rr * u.y * sigmoid_f(to_float(gr[c + 1])),
                                         v[j].z * rr * u.z * sigmoid_f(to_float(gr[c + 2])), v[j].w * rr * u.w * sigmoid_f(to_float(gr[c + 3]))));
        }
    }
}

// y = rmsnorm_group(o / (max(|n . q|, exp(-m)) + 1e-6)) * w * logistic(gate): a block per (token, group of gs columns).
// With log gates a group is a head (gs = dv; den is n . q and gates[..].z is exp(-m)); den null: nothing is divided and a
// group is whatever the caller says.  w has an entry per column.
template <typename AT, typename GT>
__global__ void __launch_bounds__(128)
memory_finish_kernel(const float* __restrict__ o, const float* __restrict__ den, const float4* __restrict__ gates,
                     const GT* __restrict__ gate, int64_t ld_gate, const float* __restrict__ w, AT* __restrict__ out,
                     int n, int gs, float eps) {
    __shared__ float scratch[32];
    wait_for_earlier_kernels();
    const int64_t t = blockIdx.x;
    const int h = blockIdx.y, H = n / gs;
    const float* row = o + t * n + (int64_t)h * gs;
    const float* wr = w + h * gs;
    const GT* gr = gate + t * ld_gate + h * gs;
    AT* orow = out + t * n + (int64_t)h * gs;
    const float inv = den ? 1.0f / (fmaxf(fabsf(den[t * H + h]), gates[t * H + h].z) + 1e-6f) : 1.0f;
    float ss = 0.f;
    for (int c = threadIdx.x; c < gs; c += blockDim.x) { const float v = row[c] * inv; ss += v * v; }
    ss = block_sum(ss, scratch);
    const float rr = inv / sqrtf(ss / (float)gs + eps);
    for (int c = threadIdx.x; c < gs; c += blockDim.x)
        orow[c] = from_float<AT>(row[c] * rr * wr[c] * sigmoid_f(to_float(gr[c])));
}

}  // namespace mem
}  // namespace mi

namespace mi {
namespace mem {

// ---------------------------------------------------------------------------
// One token per request.  A cluster of `gridDim.x` blocks per (request, head), each with a slice of the value columns:
// 16 threads side by side (VEC columns each) x 16 row groups.  Every block forms the gates and n . q itself; with log
// gates the blocks exchange their sums of squares over the cluster's network (one number each) and write the finished,
// rounded row; n and m are written by the first block after the barrier, when every block has read them.  With a fixed
// decay (whose output norm runs over all heads) the float read-out goes out and no cluster is needed.
// ---------------------------------------------------------------------------
constexpr int kDecCT = 16, kDecRG = 16, kDecMaxSlices = 8;

template <typename AT, int VEC, bool LOG>
__global__ void __launch_bounds__(256)
memory_decode_kernel(Rows in, LogGates lg, State st, const float* __restrict__ decay, const int* __restrict__ q_start,
                     const int* __restrict__ state_slot, int gate_col, const float* __restrict__ w, float eps,
                     AT* __restrict__ y, float* __restrict__ o_out, int H, int d, int dv, int cw) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float scratch[32], gsh[4], part[kDecMaxSlices];
    float* qs = sm;                         // [d] scaled queries
    float* ks = qs + d;                     // [d] keys
    float* vs = ks + d;                     // [cw] values of the slice
    float* red = vs + cw;                   // [16][cw] read-outs of the row groups
    if (LOG) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
    wait_for_earlier_kernels();
    const int b = blockIdx.z, h = blockIdx.y, c_lo = blockIdx.x * cw, nc = min(cw, dv - c_lo);
    const int tid = threadIdx.x;
    const int64_t t = q_start[b];
    float* row = st.row(state_slot[b]);
    float* S = row + st.s_off + (int64_t)h * d * dv;
    float* N = row + st.n_off + (int64_t)h * d;
    float* M = row + st.m_off + h;
    const float* pr = in.p + t * in.ld;
    for (int i = tid; i < d; i += 256) {
        float q = pr[in.q + h * d + i], k = pr[in.k + h * d + i];
        if (in.act) { q = silu_f(q); k = silu_f(k); }
        qs[i] = q * in.q_scale;
        ks[i] = k;
    }
    for (int c = tid; c < nc; c += 256) {
        const float v = pr[in.v + (int64_t)h * dv + c_lo + c];
        vs[c] = in.act ? silu_f(v) : v;
    }
    if (tid == 0) {
        if (LOG) {
            float li, lf;
            log_gates(lg, t, h, li, lf);
            const float before = *M, m = fmaxf(lf + before, li);
            gsh[0] = expf(lf + before - m);
            gsh[1] = expf(li - m);
            gsh[2] = expf(-m);
            gsh[3] = m;
        } else {
            gsh[0] = decay[h];
            gsh[1] = 1.f;
        }
    }
    __syncthreads();
    const float keep = gsh[0], write = gsh[1];
    const int ct = tid % kDecCT, rg = tid / kDecCT;
    for (int c = ct * VEC; c < nc; c += kDecCT * VEC) {
        float acc[VEC], v[VEC];
#pragma unroll
        for (int x = 0; x < VEC; ++x) { acc[x] = 0.f; v[x] = write * vs[c + x]; }
        for (int i0 = rg; i0 < d; i0 += 8 * kDecRG) {
            float s[8][VEC];
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const int i = i0 + u * kDecRG;
                if (i < d) {
                    const float* p = S + (int64_t)i * dv + c_lo + c;
                    if (VEC == 4) {
                        const float4 f = *reinterpret_cast<const float4*>(p);
                        s[u][0] = f.x; s[u][1 % VEC] = f.y; s[u][2 % VEC] = f.z; s[u][3 % VEC] = f.w;
                    } else {
                        s[u][0] = *p;
                    }
                }
            }
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const int i = i0 + u * kDecRG;
                if (i < d) {
                    const float k = ks[i], q = qs[i];
#pragma unroll
                    for (int x = 0; x < VEC; ++x) { s[u][x] = keep * s[u][x] + k * v[x]; acc[x] += s[u][x] * q; }
                    float* p = S + (int64_t)i * dv + c_lo + c;
                    if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(s[u][0], s[u][1 % VEC], s[u][2 % VEC], s[u][3 % VEC]);
                    else *p = s[u][0];
                }
            }
        }
#pragma unroll
        for (int x = 0; x < VEC; ++x) red[rg * cw + c + x] = acc[x];
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < nc; c += 256) {
        float o = 0.f;
#pragma unroll
        for (int g = 0; g < kDecRG; ++g) o += red[g * cw + c];
        if (LOG) { vs[c] = o; ss += o * o; }
        else o_out[t * H * dv + (int64_t)h * dv + c_lo + c] = o;
    }
    if constexpr (LOG) {
        float dot = 0.f;
        for (int i = tid; i < d; i += 256) dot += (keep * N[i] + write * ks[i]) * qs[i];
        ss = block_sum(ss, scratch);
        dot = block_sum(dot, scratch);
        cg::cluster_group cluster = cg::this_cluster();
        asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
        if (tid < (int)gridDim.x) *cluster.map_shared_rank(part + blockIdx.x, tid) = ss;
        cluster.sync();                         // sums have arrived; every block has read n and m
        float total = 0.f;
        for (int s = 0; s < (int)gridDim.x; ++s) total += part[s];
        const float inv = 1.0f / (fmaxf(fabsf(dot), gsh[2]) + 1e-6f);
        const float rr = inv / sqrtf(total * inv * inv / (float)dv + eps);
        for (int c = tid; c < nc; c += 256) {
            const int at = h * dv + c_lo + c;
            y[t * H * dv + at] = from_float<AT>(vs[c] * rr * w[at] * sigmoid_f(pr[gate_col + at]));
        }
        if (blockIdx.x == 0) {
            for (int i = tid; i < d; i += 256) N[i] = keep * N[i] + write * ks[i];
            if (tid == 0) *M = gsh[3];
        }
    }
}

}  // namespace mem
}  // namespace mi

// ---------------------------------------------------------------------------
// Long portions, 64 tokens (a chunk) at a time.  With F_t the sum of the log forget gates since the chunk's start the
// recurrence unrolls to
//
//   o_t = sum_(j <= t in the chunk) e^(F_t - F_j + i_j - m_t) (q_t . k_j) v_j  +  e^(F_t + m_start - m_t) S_start^T q_t
//
// (fixed decay: i = m = 0 and F_t = (t + 1) log decay).  No exponent is positive.  Three kernels:
//
//   states    U = sum_j e^(F_end - F_j + i_j - m_end) k_j v_j^T of every chunk by itself, and the chunk's whole decay
//   chain     S_start of every chunk from the one before it, element by element (the only sequential part)
//   outputs   the two sums above
//
// The projections q, k and v are the bfloat16 operands.  What the recurrence makes is float: a float factor of a
// product on the tensor cores (a weighted value, a weighted score, the state) goes in as a sum of two bfloat16 numbers,
// high part and remainder, so that it loses no more than 2^-17 of itself, and all sums are float.
// A request's chunks count from the portion's start; chunk c of request b has the index q_start[b] / 64 + b + c.
// ---------------------------------------------------------------------------
namespace mi {
namespace mem {

constexpr int kC = 64;                       // tokens per chunk
constexpr int kT = 64;                       // value columns per block
constexpr int kVP = kT + 8;                  // row stride of a value tile in shared memory

__device__ __forceinline__ uint32_t pack2(__nv_bfloat16 lo, __nv_bfloat16 hi) {
    __nv_bfloat162 v(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}
// a = high + remainder, both bfloat16
__device__ __forceinline__ void split2(float a, __nv_bfloat16& hi, __nv_bfloat16& lo) {
    hi = __float2bfloat16_rn(a);
    lo = __float2bfloat16_rn(a - __bfloat162float(hi));
}
__device__ __forceinline__ void ldmatrix_x2_trans(uint32_t& r0, uint32_t& r1, const void* smem_row) {
    const uint32_t addr = static_cast<uint32_t>(__cvta_generic_to_shared(smem_row));
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];\n" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* smem_row) {
    const uint32_t addr = static_cast<uint32_t>(__cvta_generic_to_shared(smem_row));
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* smem_row) {
    const uint32_t addr = static_cast<uint32_t>(__cvta_generic_to_shared(smem_row));
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

// Sums of the chunk's log forget gates as pairs of floats (high part, remainder), by the first warp.
__device__ __forceinline__ void chunk_log_decays(const float4* gates, int64_t t0, int nt, int H, int h, float* Fh, float* Fl) {
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x, a = 2 * lane, c = a + 1;
        const double f0 = a < nt ? (double)gates[(t0 + a) * H + h].w : 0.0;
        const double f1 = c < nt ? (double)gates[(t0 + c) * H + h].w : 0.0;
        double s = f0 + f1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s += up;
        }
        const double first = s - f1;
        Fh[a] = (float)first; Fl[a] = (float)(first - (double)Fh[a]);
        Fh[c] = (float)s; Fl[c] = (float)(s - (double)Fh[c]);
    }
}

// Projection rows in bfloat16, and what is done to them.
struct RowsB {
    const __nv_bfloat16* p;
    int64_t ld;
    int q, k, v;
    int act;
    float q_scale;
    int vec;                // rows, columns and heads on 16-byte boundaries
};

__device__ __forceinline__ void copy_async_16b(void* smem_dst, const void* src) {
    const uint32_t dst = static_cast<uint32_t>(__cvta_generic_to_shared(smem_dst));
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(src));
}
__device__ __forceinline__ void copy_async_wait_all() { asm volatile("cp.async.wait_all;\n" ::: "memory"); }

// eight neighbouring numbers of a row through the activation (zeros from column n on)
__device__ __forceinline__ uint4 load8(const __nv_bfloat16* p, int n, int act, bool vec) {
    uint4 r = make_uint4(0u, 0u, 0u, 0u);
    __nv_bfloat16* e = reinterpret_cast<__nv_bfloat16*>(&r);
    if (vec && n >= 8) r = *reinterpret_cast<const uint4*>(p);
    else {
#pragma unroll
        for (int x = 0; x < 8; ++x) if (x < n) e[x] = p[x];
    }
    if (act) {
#pragma unroll
        for (int x = 0; x < 8; ++x) { const float f = __bfloat162float(e[x]); e[x] = __float2bfloat16_rn(__fdividef(f, 1.0f + __expf(-f))); }
    }
    return r;
}

// 64 rows of `width` columns (padded to wp, a multiple of 8) into shared memory; rows from nt on are zeros.  Without an
// activation, copies that nothing has to touch are left in flight (copy_async_wait_all before the barrier).
__device__ __forceinline__ void fill_rows(__nv_bfloat16* dst, int pitch, const __nv_bfloat16* src, int64_t ld, int width, int wp,
                                          int nt, int act, bool vec) {
    const int w8 = wp / 8;
    for (int idx = threadIdx.x; idx < kC * w8; idx += blockDim.x) {
        const int j = idx / w8, i = 8 * (idx - j * w8);
        __nv_bfloat16* d = dst + j * pitch + i;
        if (j < nt && vec && !act && i + 8 <= width) copy_async_16b(d, src + j * ld + i);
        else *reinterpret_cast<uint4*>(d) = j < nt ? load8(src + j * ld + i, width - i, act, vec) : make_uint4(0u, 0u, 0u, 0u);
    }
}

// U [chunk][H][d][dvp] (dvp: dv rounded up to 8, zeros beyond dv), Un [chunk][H][d] (log gates), keepc [chunk][H].  A block
// of 4 warps takes a value tile of 64 columns of one (chunk, head).  The weights go into the values, w_j v_j, as high part
// and remainder: a tile's values are its own, while its keys serve every tile of the head.  dp = d rounded up to 16.
template <bool LOG>
__global__ void __launch_bounds__(128)
memory_chunk_states_kernel(RowsB in, const float4* __restrict__ gates, const float4* __restrict__ logs,
                           const float* __restrict__ decay, const int* __restrict__ q_start, float* __restrict__ U,
                           float* __restrict__ Un, float* __restrict__ keepc, int H, int d, int dv, int dvp, int dp,
                           int tiles) {
    extern __shared__ __align__(16) unsigned char raw[];
    __shared__ float Fh[kC], Fl[kC], wj[kC];
    wait_for_earlier_kernels();
    const int b = blockIdx.z, h = blockIdx.y / tiles, tile = blockIdx.y % tiles, c = blockIdx.x;
    const int q0 = q_start[b], n = q_start[b + 1] - q0;
    if (c * kC >= n) return;
    const int nt = min(kC, n - c * kC);
    const int64_t t0 = q0 + c * kC, at = (int64_t)(q0 / kC + b + c) * H + h;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int kp = dp + 8;
    __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(raw);      // [64][kp] keys
    __nv_bfloat16* Vh = Ks + kC * kp;                               // [64][kVP] weighted values, high parts
    __nv_bfloat16* Vl = Vh + kC * kVP;                              // remainders
    const int v_lo = tile * kT, nv = min(kT, dv - v_lo);
    fill_rows(Ks, kp, in.p + t0 * in.ld + in.k + h * d, in.ld, d, dp, nt, in.act, in.vec);
    if (LOG) {
        chunk_log_decays(gates, t0, nt, H, h, Fh, Fl);
        __syncthreads();
        if (tid < kC) {
            const float4 lg = tid < nt ? logs[(t0 + tid) * H + h] : make_float4(0.f, 0.f, 0.f, 0.f);
            const float m_end = logs[(t0 + nt - 1) * H + h].y;
            wj[tid] = tid < nt ? expf((Fh[nt - 1] - Fh[tid]) + (Fl[nt - 1] - Fl[tid]) + (lg.x - m_end)) : 0.f;
            if (tid == 0 && tile == 0) keepc[at] = expf(Fh[nt - 1] + (lg.z - m_end));
        }
    } else if (tid < kC) {
        const float ld = fmaxf(logf(decay[h]), -1e30f);
        wj[tid] = tid < nt ? expf((float)(nt - 1 - tid) * ld) : 0.f;
        if (tid == 0 && tile == 0) keepc[at] = expf((float)nt * ld);
    }
    __syncthreads();
    for (int idx = tid; idx < kC * (kT / 8); idx += 128) {
        const int j = idx / (kT / 8), i = 8 * (idx % (kT / 8));
        uint4 v = make_uint4(0u, 0u, 0u, 0u), lo8;
        if (j < nt) v = load8(in.p + (t0 + j) * in.ld + in.v + (int64_t)h * dv + v_lo + i, nv - i, in.act, in.vec);
        __nv_bfloat16* hi = reinterpret_cast<__nv_bfloat16*>(&v);
        __nv_bfloat16* lo = reinterpret_cast<__nv_bfloat16*>(&lo8);
        const float w = wj[j];
#pragma unroll
        for (int x = 0; x < 8; ++x) { const float f = w * __bfloat162float(hi[x]); split2(f, hi[x], lo[x]); }
        *reinterpret_cast<uint4*>(Vh + j * kVP + i) = v;
        *reinterpret_cast<uint4*>(Vl + j * kVP + i) = lo8;
    }
    copy_async_wait_all();
    __syncthreads();
    float* Ub = U + at * d * dvp + v_lo;
    const int nvp = min(kT, dvp - v_lo);
    for (int mt = warp; mt < dp / 16; mt += 4) {
        float acc[8][4];
#pragma unroll
        for (int x = 0; x < 8; ++x) acc[x][0] = acc[x][1] = acc[x][2] = acc[x][3] = 0.f;
#pragma unroll
        for (int kk = 0; kk < kC / 16; ++kk) {
            // A[i][j] = k_j[i]: the keys lie token by token, so the fragments are fetched transposed
            uint32_t a[4];
            ldmatrix_x4_trans(a, Ks + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * kp + mt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int x = 0; x < 8; x += 2) {
                uint32_t bh[4], bl[4];                    // two neighbouring tiles of 8 columns
                const int off = (kk * 16 + (lane & 15)) * kVP + (x + (lane >> 4)) * 8;
                ldmatrix_x4_trans(bh, Vh + off);
                ldmatrix_x4_trans(bl, Vl + off);
                mma_bf16_16816(acc[x], a[0], a[1], a[2], a[3], bh[0], bh[1]);
                mma_bf16_16816(acc[x], a[0], a[1], a[2], a[3], bl[0], bl[1]);
                mma_bf16_16816(acc[x + 1], a[0], a[1], a[2], a[3], bh[2], bh[3]);
                mma_bf16_16816(acc[x + 1], a[0], a[1], a[2], a[3], bl[2], bl[3]);
            }
        }
        const int r0 = mt * 16 + (lane >> 2), c2 = (lane & 3) * 2;
#pragma unroll
        for (int x = 0; x < 8; ++x) {
            const int col = x * 8 + c2;
            if (col < nvp) {
                if (r0 < d) *reinterpret_cast<float2*>(Ub + (int64_t)r0 * dvp + col) = make_float2(acc[x][0], acc[x][1]);
                if (r0 + 8 < d) *reinterpret_cast<float2*>(Ub + (int64_t)(r0 + 8) * dvp + col) = make_float2(acc[x][2], acc[x][3]);
            }
        }
    }
    if (LOG && tile == 0)
        for (int i = tid; i < d; i += 128) {
            float s = 0.f;
            for (int j = 0; j < nt; ++j) s += wj[j] * __bfloat162float(Ks[j * kp + i]);
            Un[at * d + i] = s;
        }
}

// S_start[0] = the request's state, S_start[c + 1] = keepc[c] S_start[c] + U[c], a thread per eight columns of a row of S;
// what follows the last chunk is the request's new state.  S_start[c] takes the place of U[c] once that has been read, as
// eight high parts and eight remainders in bfloat16: what the outputs' products take.  With Un the last block of every
// head chains n in the same way (it stays float).
__global__ void __launch_bounds__(256)
memory_chunk_chain_kernel(float* __restrict__ U, float* __restrict__ Un, const float* __restrict__ keepc,
                          float* __restrict__ state, int64_t state_stride, int64_t off, int64_t n_off,
                          const int* __restrict__ q_start, const int* __restrict__ state_slot, int H, int d, int dv, int dvp) {
    wait_for_earlier_kernels();
    const int b = blockIdx.z, h = blockIdx.y;
    if (Un && blockIdx.x == gridDim.x - 1) {
        const int i = threadIdx.x, q0 = q_start[b], n = q_start[b + 1] - q0;        // (keys of at most 256 numbers)
        if (i >= d || n <= 0) return;
        const int chunks = (n + kC - 1) / kC;
        const int64_t first = (int64_t)(q0 / kC + b) * H + h;
        float* S = state + (int64_t)state_slot[b] * state_stride + n_off + (int64_t)h * d + i;
        float cur = *S;
        for (int c0 = 0; c0 < chunks; c0 += 8) {
            float u[8], keep[8];
#pragma unroll
            for (int a = 0; a < 8; ++a) {
                const int64_t at = first + (int64_t)min(c0 + a, chunks - 1) * H;
                u[a] = Un[at * d + i];
                keep[a] = keepc[at];
            }
#pragma unroll
            for (int a = 0; a < 8; ++a)
                if (c0 + a < chunks) { Un[(first + (int64_t)(c0 + a) * H) * d + i] = cur; cur = keep[a] * cur + u[a]; }
        }
        *S = cur;
        return;
    }
    const int e = blockIdx.x * blockDim.x + threadIdx.x, groups = dvp / 8;
    const int q0 = q_start[b], n = q_start[b + 1] - q0;
    if (e >= d * groups || n <= 0) return;
    const int i = e / groups, c8 = 8 * (e - i * groups);
    const int chunks = (n + kC - 1) / kC;
    const int64_t first = (int64_t)(q0 / kC + b) * H + h, size = (int64_t)d * dvp;
    float* S = state + (int64_t)state_slot[b] * state_stride + off + (int64_t)h * d * dv + (int64_t)i * dv + c8;
    float cur[8];
#pragma unroll
    for (int x = 0; x < 8; ++x) cur[x] = c8 + x < dv ? S[x] : 0.f;
    float* base = U + first * size + (int64_t)i * dvp + c8;
    const int64_t step = H * size;
    constexpr int AHEAD = 2;
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        float4 u[AHEAD][2];
        float keep[AHEAD];
#pragma unroll
        for (int a = 0; a < AHEAD; ++a)
            if (c0 + a < chunks) {
                const float4* p = reinterpret_cast<const float4*>(base + (c0 + a) * step);
                u[a][0] = p[0];
                u[a][1] = p[1];
                keep[a] = keepc[first + (int64_t)(c0 + a) * H];
            }
#pragma unroll
        for (int a = 0; a < AHEAD; ++a)
            if (c0 + a < chunks) {
                uint4 out[2];
                __nv_bfloat16* hl = reinterpret_cast<__nv_bfloat16*>(out);
#pragma unroll
                for (int x = 0; x < 8; ++x) split2(cur[x], hl[x], hl[8 + x]);
                uint4* p = reinterpret_cast<uint4*>(base + (c0 + a) * step);
                p[0] = out[0];
                p[1] = out[1];
                const float* uu = reinterpret_cast<const float*>(u[a]);
#pragma unroll
                for (int x = 0; x < 8; ++x) cur[x] = keep[a] * cur[x] + uu[x];
            }
    }
#pragma unroll
    for (int x = 0; x < 8; ++x) if (c8 + x < dv) S[x] = cur[x];
}

// Read-outs of a chunk.  Block = 8 warps: warp w owns the tokens 16 (w % 4) .. + 15 of the chunk and half of a value tile of
// 64 columns; the block walks over `per` tiles of its head.  The weighted scores are formed once, as high part and
// remainder in registers; a tile then costs its start state (which takes the place of the keys in shared memory) and its
// values.
template <bool LOG>
__global__ void __launch_bounds__(256)
memory_chunk_outputs_kernel(RowsB in, const float4* __restrict__ gates, const float4* __restrict__ logs,
                            const float* __restrict__ decay, const int* __restrict__ q_start,
                            const float* __restrict__ S0, const float* __restrict__ N0, float* __restrict__ out,
                            float* __restrict__ den, int H, int d, int dv, int dvp, int dp, int tiles, int per, int groups) {
    extern __shared__ __align__(16) unsigned char raw[];
    __shared__ float Fh[kC], Fl[kC], ij[kC], mj[kC], inter[kC], pw[kC + 1];
    wait_for_earlier_kernels();
    const int b = blockIdx.z, h = blockIdx.y / groups, group = blockIdx.y % groups, c = blockIdx.x;
    const int q0 = q_start[b], n = q_start[b + 1] - q0;
    if (c * kC >= n) return;
    const int nt = min(kC, n - c * kC);
    const int64_t t0 = q0 + c * kC, at = (int64_t)(q0 / kC + b + c) * H + h;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, wr = warp & 3, wc = warp >> 2;
    const int kp = dp + 8;
    constexpr int SPB = kT * 4 + 16;                                // bytes of a row of the start state's tile
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(raw);      // [64][kp]
    __nv_bfloat16* Vs = Qs + kC * kp;                               // [64][kVP]
    __nv_bfloat16* Ks = Vs + kC * kVP;                              // [64][kp], then [dp] rows of the start state
    unsigned char* Ss = reinterpret_cast<unsigned char*>(Ks);
    fill_rows(Qs, kp, in.p + t0 * in.ld + in.q + h * d, in.ld, d, dp, nt, in.act, in.vec);
    fill_rows(Ks, kp, in.p + t0 * in.ld + in.k + h * d, in.ld, d, dp, nt, in.act, in.vec);
    if (LOG) {
        chunk_log_decays(gates, t0, nt, H, h, Fh, Fl);
        __syncthreads();
        if (tid < kC) {
            const float4 lg = tid < nt ? logs[(t0 + tid) * H + h] : make_float4(0.f, 0.f, 0.f, 0.f);
            ij[tid] = lg.x;
            mj[tid] = lg.y;
            inter[tid] = tid < nt ? expf(Fh[tid] + (logs[t0 * H + h].z - lg.y)) : 0.f;
        }
    } else if (tid <= kC) {
        pw[tid] = expf((float)tid * fmaxf(logf(decay[h]), -1e30f));
    }
    copy_async_wait_all();
    __syncthreads();
    const int r0 = lane >> 2, c2 = (lane & 3) * 2;
    const int ta = wr * 16 + r0, tb = ta + 8;               // this thread's two tokens
    uint32_t wh[4][4], wl[4][4];                            // weighted scores as fragments, 16 keys each
    const float ia = (LOG ? inter[ta] : pw[ta + 1]) * in.q_scale, ib = (LOG ? inter[tb] : pw[tb + 1]) * in.q_scale;
    {
        float sc[8][4];
#pragma unroll
        for (int x = 0; x < 8; ++x) sc[x][0] = sc[x][1] = sc[x][2] = sc[x][3] = 0.f;
        for (int ks = 0; ks < dp; ks += 16) {
            uint32_t a[4];
            ldmatrix_x4(a, Qs + (wr * 16 + (lane & 15)) * kp + ks + (lane >> 4) * 8);
#pragma unroll
            for (int x = 0; x < 8; x += 2) {
                if (x < 2 * wr + 2) {                       // keys up to this warp's last token
                    uint32_t k4[4];                         // (keys 8x .. + 7, + 8 .. + 15) x (columns ks .. + 7, + 8 .. + 15)
                    ldmatrix_x4(k4, Ks + (x * 8 + (lane >> 4) * 8 + (lane & 7)) * kp + ks + ((lane >> 3) & 1) * 8);
                    mma_bf16_16816(sc[x], a[0], a[1], a[2], a[3], k4[0], k4[1]);
                    mma_bf16_16816(sc[x + 1], a[0], a[1], a[2], a[3], k4[2], k4[3]);
                }
            }
        }
        float suma = 0.f, sumb = 0.f;
#pragma unroll
        for (int x = 0; x < 8; ++x) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int j = x * 8 + c2 + (e & 1), t = e < 2 ? ta : tb;
                float wgt = 0.f;
                if (j <= t) wgt = LOG ? expf((Fh[t] - Fh[j]) + (Fl[t] - Fl[j]) + (ij[j] - mj[t])) : pw[t - j];
                sc[x][e] *= wgt * in.q_scale;
            }
            suma += sc[x][0] + sc[x][1];
            sumb += sc[x][2] + sc[x][3];
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk)
#pragma unroll
            for (int f = 0; f < 4; ++f) {
                // fragment f: rows ta (0, 2) and tb (1, 3), keys c2, c2 + 1 of the first (0, 1) and second eight (2, 3)
                __nv_bfloat16 h0, l0, h1, l1;
                split2(sc[2 * kk + (f >> 1)][2 * (f & 1)], h0, l0);
                split2(sc[2 * kk + (f >> 1)][2 * (f & 1) + 1], h1, l1);
                wh[kk][f] = pack2(h0, h1);
                wl[kk][f] = pack2(l0, l1);
            }
        if (LOG && group == 0 && wc == 0) {
            // n . q: the weights' sum and what the start of the chunk brought
            suma += __shfl_xor_sync(0xffffffffu, suma, 1); suma += __shfl_xor_sync(0xffffffffu, suma, 2);
            sumb += __shfl_xor_sync(0xffffffffu, sumb, 1); sumb += __shfl_xor_sync(0xffffffffu, sumb, 2);
            const float* nb = N0 + at * d;
            float da = 0.f, db = 0.f;
            for (int i = lane & 3; i < d; i += 4) {
                const float x = nb[i];
                da += x * __bfloat162float(Qs[ta * kp + i]);
                db += x * __bfloat162float(Qs[tb * kp + i]);
            }
            da += __shfl_xor_sync(0xffffffffu, da, 1); da += __shfl_xor_sync(0xffffffffu, da, 2);
            db += __shfl_xor_sync(0xffffffffu, db, 1); db += __shfl_xor_sync(0xffffffffu, db, 2);
            if ((lane & 3) == 0) {
                if (ta < nt) den[(t0 + ta) * H + h] = suma + ia * da;
                if (tb < nt) den[(t0 + tb) * H + h] = sumb + ib * db;
            }
        }
    }
    for (int tile = group * per; tile < min(tiles, (group + 1) * per); ++tile) {
        const int v_lo = tile * kT, nv = min(kT, dv - v_lo), nvp = min(kT, dvp - v_lo);
        __syncthreads();                                    // the keys, or the tile before, have been read
        const float* Sb = S0 + at * d * dvp + v_lo;
        for (int idx = tid; idx < dp * (kT / 4); idx += 256) {
            const int i = idx / (kT / 4), q4 = 4 * (idx % (kT / 4));
            unsigned char* dst = Ss + i * SPB + q4 * 4;
            if (i < d && q4 < nvp) copy_async_16b(dst, Sb + (int64_t)i * dvp + q4);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0u, 0u, 0u, 0u);
        }
        fill_rows(Vs, kVP, in.p + t0 * in.ld + in.v + (int64_t)h * dv + v_lo, in.ld, nv, kT, nt, in.act, in.vec);
        copy_async_wait_all();
        __syncthreads();
        float acc[4][4];
#pragma unroll
        for (int x = 0; x < 4; ++x) acc[x][0] = acc[x][1] = acc[x][2] = acc[x][3] = 0.f;
        for (int ks = 0; ks < dp; ks += 16) {
            uint32_t a[4];
            ldmatrix_x4(a, Qs + (wr * 16 + (lane & 15)) * kp + ks + (lane >> 4) * 8);
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                uint32_t s4[4];                             // eight columns: high parts, then remainders
                ldmatrix_x4_trans(s4, Ss + (ks + (lane & 15)) * SPB + (wc * 4 + x) * 32 + (lane >> 4) * 16);
                mma_bf16_16816(acc[x], a[0], a[1], a[2], a[3], s4[0], s4[1]);
                mma_bf16_16816(acc[x], a[0], a[1], a[2], a[3], s4[2], s4[3]);
            }
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) { acc[x][0] *= ia; acc[x][1] *= ia; acc[x][2] *= ib; acc[x][3] *= ib; }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            if (kk <= wr) {
#pragma unroll
                for (int x = 0; x < 4; x += 2) {
                    uint32_t b4[4];
                    ldmatrix_x4_trans(b4, Vs + (kk * 16 + (lane & 15)) * kVP + (wc * 4 + x + (lane >> 4)) * 8);
                    mma_bf16_16816(acc[x], wh[kk][0], wh[kk][1], wh[kk][2], wh[kk][3], b4[0], b4[1]);
                    mma_bf16_16816(acc[x], wl[kk][0], wl[kk][1], wl[kk][2], wl[kk][3], b4[0], b4[1]);
                    mma_bf16_16816(acc[x + 1], wh[kk][0], wh[kk][1], wh[kk][2], wh[kk][3], b4[2], b4[3]);
                    mma_bf16_16816(acc[x + 1], wl[kk][0], wl[kk][1], wl[kk][2], wl[kk][3], b4[2], b4[3]);
                }
            }
        }
        float* ob = out + t0 * H * dv + (int64_t)h * dv + v_lo;
        const bool pair = (dv & 1) == 0;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int col = (wc * 4 + x) * 8 + c2;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = e ? tb : ta;
                if (t < nt) {
                    float* p = ob + (int64_t)t * H * dv + col;
                    if (pair && col + 1 < nv) *reinterpret_cast<float2*>(p) = make_float2(acc[x][2 * e], acc[x][2 * e + 1]);
                    else { if (col < nv) p[0] = acc[x][2 * e]; if (col + 1 < nv) p[1] = acc[x][2 * e + 1]; }
                }
            }
        }
    }
}

}  // namespace mem
}  // namespace mi

using namespace mi;

extern "C" {

static bool bad_memory(int B, int H, int d, int dv, int64_t ld) {
    if (d < 1 || d > 256 || dv < 1 || H < 1 || H > 65535 || B > 65535 || ld < 1) {
        set_last_error("matrix memory: %d heads of key size %d (at most 256) and value size %d, batch %d", H, d, dv, B);
        return true;
    }
    return false;
}

// The log gates of a step and the chain of their running maximum (state: float rows, m [H] at m_off).  gates and logs
// hold T * H * 4 floats (logs may be null).  scan: the chain composed in a tree (see memory_gates_kernel).
int mi_memory_gates(const float* proj, int ld, int col_i, int col_f, const float* bi, const float* bf, float cap,
                    float* state, int64_t stride, int64_t m_off, const int* q_start, const int* state_slot, float* gates,
                    float* logs, int B, int H, int scan, cudaStream_t stream) {
    if (B <= 0) return kOk;
    if (bad_memory(B, H, 1, 1, ld)) return kBadShape;
    if (!(cap > 0.f)) { set_last_error("matrix memory: gates capped at %g", (double)cap); return kBadShape; }
    const mem::LogGates lg = {proj, ld, col_i, col_f, bi, bf, cap};
    const mem::State st = {state, stride, 0, 0, m_off};
    if (scan)
        launch_dependent(mem::memory_gates_kernel<true>, dim3(H, B), dim3(256), 0, stream, lg, st, q_start, state_slot,
                         (float4*)gates, (float4*)logs, H);
    else
        launch_dependent(mem::memory_gates_kernel<false>, dim3(H, B), dim3(256), 0, stream, lg, st, q_start, state_slot,
                         (float4*)gates, (float4*)logs, H);
    return finish_launch("memory_gates");
}

// gates: as mi_memory_gates leaves them, or null with decay [H].  out [T, H*dv]; den [T, H] (with gates).
int mi_memory_walk(const float* proj, int ld, int col_q, int col_k, int col_v, int act, float q_scale, float* state,
                   int64_t stride, int64_t s_off, int64_t n_off, const float* gates, const float* decay,
                   const int* q_start, const int* state_slot, float* out, float* den, int B, int H, int d, int dv,
                   cudaStream_t stream) {
    if (B <= 0) return kOk;
    if (bad_memory(B, H, d, dv, ld)) return kBadShape;
    if ((gates == nullptr) == (decay == nullptr) || (gates && !den)) {
        set_last_error("matrix memory: either log gates (with a place for n . q) or fixed decays");
        return kBadShape;
    }
    const mem::Rows in = {proj, ld, col_q, col_k, col_v, act, q_scale};
    const mem::State st = {state, stride, s_off, n_off, 0};
    const int vec = d % 4 == 0 && ld % 4 == 0 && col_q % 4 == 0 && col_k % 4 == 0 && (reinterpret_cast<uintptr_t>(proj) & 15) == 0;
    const dim3 grid((dv + (gates ? 1 : 0) + mem::kCols - 1) / mem::kCols, H, B);
#define MI_WALK(RP, LOG)                                                                                              \
    do {                                                                                                              \
        const size_t smem = sizeof(float) * (2 * mem::kChunk * (2 * RP * mem::kLanes + mem::kCols + 4) + mem::kChunk * mem::kCols); \
        cudaFuncSetAttribute(mem::memory_walk_kernel<RP, LOG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        launch_dependent(mem::memory_walk_kernel<RP, LOG>, grid, dim3(128), smem, stream, in, st, (const float4*)gates, \
                         decay, q_start, state_slot, out, den, H, d, dv, vec);                                        \
    } while (0)
    if (gates) { if (d <= 64) MI_WALK(8, true); else if (d <= 128) MI_WALK(16, true); else MI_WALK(32, true); }
    else { if (d <= 64) MI_WALK(8, false); else if (d <= 128) MI_WALK(16, false); else MI_WALK(32, false); }
#undef MI_WALK
    return finish_launch("memory_walk");
}

int mi_memory_chunk_tokens() { return mem::kC; }

// floats of a row of the chunks' scratch U for a value size
int mi_memory_chunk_value_pitch(int dv) { return (dv + 7) / 8 * 8; }

// The same over chunks of 64 tokens on the tensor cores: q, k and v as columns of bfloat16 rows.  gates, logs: as
// mi_memory_gates leaves them, or null with decay.  U: (T / 64 + B) * H * d * mi_memory_chunk_value_pitch(dv) floats of
// scratch, Un: (..) * H * d (with gates), keepc: (..) * H.
int mi_memory_chunks(const void* proj, int ld, int col_q, int col_k, int col_v, int act, float q_scale, float* state,
                     int64_t stride, int64_t s_off, int64_t n_off, const float* gates, const float* logs,
                     const float* decay, const int* q_start, const int* state_slot, float* out, float* den, float* U,
                     float* Un, float* keepc, int B, int max_q_len, int H, int d, int dv, cudaStream_t stream) {
    if (B <= 0 || max_q_len <= 0) return kOk;
    if (bad_memory(B, H, d, dv, ld)) return kBadShape;
    const int tiles = (dv + mem::kT - 1) / mem::kT, dp = (d + 15) / 16 * 16, chunks = (max_q_len + mem::kC - 1) / mem::kC;
    const int dvp = mi_memory_chunk_value_pitch(dv);
    if ((gates == nullptr) == (decay == nullptr) || (gates && (!den || !logs || !Un)) || !U || !keepc ||
        (reinterpret_cast<uintptr_t>(U) & 15) || (int64_t)H * tiles > 65535) {
        set_last_error("matrix memory in chunks: log gates or fixed decays with their scratch; %d heads x %d value tiles", H, tiles);
        return kBadShape;
    }
    const int vec = d % 8 == 0 && dv % 8 == 0 && ld % 8 == 0 && col_q % 8 == 0 && col_k % 8 == 0 && col_v % 8 == 0 &&
                    (reinterpret_cast<uintptr_t>(proj) & 15) == 0;
    const mem::RowsB in = {(const __nv_bfloat16*)proj, ld, col_q, col_k, col_v, act, q_scale, vec};
    // value tiles a block of the outputs walks over: as many as leave two blocks per SM
    const int64_t blocks = (int64_t)chunks * H * tiles * B;
    int per = (int)(blocks / 296);
    per = per < 1 ? 1 : (per > tiles ? tiles : per);
    const int groups = (tiles + per - 1) / per;
    const size_t rows_bytes = (size_t)mem::kC * (dp + 8) * 2, v_bytes = (size_t)mem::kC * mem::kVP * 2;
    const size_t s_bytes = (size_t)dp * (mem::kT * 4 + 16);
    const size_t smem_s = rows_bytes + 2 * v_bytes;
    const size_t smem_o = rows_bytes + v_bytes + (rows_bytes > s_bytes ? rows_bytes : s_bytes);
#define MI_CHUNKS(LOG)                                                                                                 \
    do {                                                                                                               \
        cudaFuncSetAttribute(mem::memory_chunk_states_kernel<LOG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_s); \
        cudaFuncSetAttribute(mem::memory_chunk_outputs_kernel<LOG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_o); \
        launch_dependent(mem::memory_chunk_states_kernel<LOG>, dim3(chunks, H * tiles, B), dim3(128), smem_s, stream, in, \
                         (const float4*)gates, (const float4*)logs, decay, q_start, U, Un, keepc, H, d, dv, dvp, dp, tiles); \
        launch_dependent(mem::memory_chunk_chain_kernel, dim3((d * (dvp / 8) + 255) / 256 + (LOG ? 1 : 0), H, B), dim3(256), \
                         0, stream, U, LOG ? Un : nullptr, (const float*)keepc, state, stride, s_off, n_off, q_start,  \
                         state_slot, H, d, dv, dvp);                                                                   \
        launch_dependent(mem::memory_chunk_outputs_kernel<LOG>, dim3(chunks, H * groups, B), dim3(256), smem_o, stream, in, \
                         (const float4*)gates, (const float4*)logs, decay, q_start, (const float*)U, (const float*)Un, out, \
                         den, H, d, dv, dvp, dp, tiles, per, groups);                                                  \
    } while (0)
    if (gates) MI_CHUNKS(true); else MI_CHUNKS(false);
#undef MI_CHUNKS
    return finish_launch("memory_chunks", 3);
}

// out [T, n] = rmsnorm over groups of gs columns of o / (max(|den|, exp(-m)) + 1e-6), times w [n], times logistic(gate);
// den and gates null: nothing is divided.  gate: rows of ld_gate numbers of the type gdtype.
int mi_memory_finish(const float* o, const float* den, const float* gates, const void* gate, int gdtype, int ld_gate,
                     const float* w, void* out, int adtype, int T, int n, int gs, float eps, cudaStream_t stream) {
    if (T <= 0) return kOk;
    if (gs < 1 || n % gs || n / gs > 65535 || (den == nullptr) != (gates == nullptr)) {
        set_last_error("matrix memory: %d columns in groups of %d", n, gs);
        return kBadShape;
    }
    const bool vec = gs % 4 == 0 && gs <= 8192 &&
                     ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    const int64_t total = (int64_t)T * (n / gs);
#define MI_FINISH_VEC(VPT, ONE)                                                                                       \
    MI_DISPATCH_2(adtype, AT, gdtype, GT,                                                                             \
        launch_dependent(mem::memory_finish_vec_kernel<AT, GT, VPT, ONE>, dim3((unsigned)(ONE ? (total + 7) / 8 : total)), \
                         dim3(256), 0, stream, o, den, (const float4*)gates, (const GT*)gate, ld_gate, w, (AT*)out, n, gs, \
                         eps, total))
    if (vec) {
        if (gs <= 128) MI_FINISH_VEC(1, true);
        else if (gs <= 256) MI_FINISH_VEC(2, true);
        else if (gs <= 512) MI_FINISH_VEC(4, true);
        else if (gs <= 2048) MI_FINISH_VEC(2, false);
        else if (gs <= 4096) MI_FINISH_VEC(4, false);
        else MI_FINISH_VEC(8, false);
#undef MI_FINISH_VEC
        return finish_launch("memory_finish");
    }
    int threads = 32;
    while (threads < gs && threads < 128) threads *= 2;
    MI_DISPATCH_2(adtype, AT, gdtype, GT,
        launch_dependent(mem::memory_finish_kernel<AT, GT>, dim3(T, n / gs), dim3(threads), 0, stream, o, den,
                         (const float4*)gates, (const GT*)gate, ld_gate, w, (AT*)out, n, gs, eps));
    return finish_launch("memory_finish");
}

// One token per request (checked by the caller).  Log gates (decay null): y [T, H*dv] in the type `adtype` is the
// finished row; fixed decays: o_out [T, H*dv] float is the read-out.
int mi_memory_decode(const float* proj, int ld, int col_q, int col_k, int col_v, int act, float q_scale, int col_i,
                     int col_f, const float* bi, const float* bf, float cap, float* state, int64_t stride, int64_t s_off,
                     int64_t n_off, int64_t m_off, const float* decay, const int* q_start, const int* state_slot,
                     int col_gate, const float* w, float eps, void* y, int adtype, float* o_out, int B, int H, int d,
                     int dv, cudaStream_t stream) {
    if (B <= 0) return kOk;
    if (bad_memory(B, H, d, dv, ld)) return kBadShape;
    if (decay ? !o_out : (!y || !w || !bi || !bf || !(cap > 0.f))) {
        set_last_error("matrix memory of a decode step: an operand is missing");
        return kBadShape;
    }
    const bool v4 = dv % 4 == 0 && s_off % 4 == 0 && stride % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
    // slices of at least 32 columns: enough blocks for the device at small batches, at most a cluster of eight
    int slices = (dv + 31) / 32;
    if (slices > mem::kDecMaxSlices) slices = mem::kDecMaxSlices;
    int cw = (dv + slices - 1) / slices;
    cw = (cw + 3) / 4 * 4;
    slices = (dv + cw - 1) / cw;
    const size_t smem = sizeof(float) * (2 * d + cw + (size_t)mem::kDecRG * cw);
    if (smem > 200 * 1024) { set_last_error("matrix memory of a decode step: value size %d", dv); return kBadShape; }
    const mem::Rows in = {proj, ld, col_q, col_k, col_v, act, q_scale};
    const mem::LogGates lg = {proj, ld, col_i, col_f, bi, bf, cap};
    const mem::State st = {state, stride, s_off, n_off, m_off};
    cudaLaunchConfig_t lc = {};
    lc.gridDim = dim3(slices, H, B);
    lc.blockDim = dim3(256);
    lc.dynamicSmemBytes = smem;
    lc.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = slices;
    attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = 1;
    lc.attrs = dependent_launch_enabled() ? attr : attr + 1;
    lc.numAttrs = (dependent_launch_enabled() ? 1 : 0) + (decay ? 0 : 1);
#define MI_DECODE(VEC, LOG)                                                                                           \
    MI_DISPATCH_1(adtype, AT, {                                                                                       \
        if (smem > 48 * 1024)                                                                                         \
            cudaFuncSetAttribute(mem::memory_decode_kernel<AT, VEC, LOG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        (void)cudaLaunchKernelEx(&lc, mem::memory_decode_kernel<AT, VEC, LOG>, in, lg, st, decay, q_start, state_slot, \
                                 col_gate, w, eps, (AT*)y, o_out, H, d, dv, cw);                                      \
    })
    if (decay) { if (v4) MI_DECODE(4, false); else MI_DECODE(1, false); }
    else { if (v4) MI_DECODE(4, true); else MI_DECODE(1, true); }
#undef MI_DECODE
    return finish_launch("memory_decode");
}

}  // extern "C"
