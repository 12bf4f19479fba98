// A linear recurrence per channel with gates that are products of the channels of one part (real-gated linear recurrent
// unit):  with u the output of a short convolution over time, split into `blocks` equal parts of n channels,
//
//   r = logistic(A_b u_b + ra),  i = logistic(I_b u_b + ri)        A_b, I_b [n, n], one pair per part
//   log a = rate r,  rate = -8 softplus(lam),  S_t = a S_(t-1) + sqrt(1 - a^2) i u,  out = S gelu(y + bias)
//
//   lru_gates_tc   both gates' products on the tensor cores, gates and decays in the epilogue (bfloat16 path).  u is
//                  float: it enters as the sum of three bfloat16 numbers, which holds all 24 bits of it, the matrices
//                  are bfloat16 as they are, and the sums are float, so the products are those of 32-bit arithmetic
//   lru_prepare    gates and decays from products that another kernel made (float32 path)
//   lru_scan       the recurrence: a thread per channel, in one piece (float32 path, short portions) or in segments of
//                  64 tokens side by side whose carries are chained between two passes; the second branch's gelu and
//                  the product of the two on the way out
//   lru_decode     one token per request: convolution, gates, recurrence, output and both states in one launch
//
// All of it is float arithmetic.  State of a slot: S [W] at `s_off`, the last taps-1 inputs of the convolution
// (time-major) at `c_off`.

#include <cooperative_groups.h>

#include "common.cuh"

namespace cg = cooperative_groups;

namespace mi {
namespace lru {

constexpr int kMaxTaps = 8;
constexpr int kSeg = 64;                     // tokens per segment

__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// decay and drive of a channel from its gates' inputs and its rate (-8 softplus(lam)); 1 - a^2 = -(e^(2 log a) - 1) without cancellation
__device__ __forceinline__ void decay_drive(float zr, float zi, float rate, float u, float& a, float& x) {
    const float log_a = rate * sigmoid_f(zr);
    a = expf(log_a);
    x = sqrtf(-expm1f(2.0f * log_a)) * sigmoid_f(zi) * u;
}

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* smem_row) {
    const uint32_t addr = static_cast<uint32_t>(__cvta_generic_to_shared(smem_row));
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

// Block = 8 warps: 64 tokens x 64 output channels of one part, both gates (warp w: 16 tokens, 32 channels).  ra, ri
// [blocks][n][n] bfloat16 (out, in).  The inner dimension goes by in slices of 32: while one slice is multiplied, the next
// one's matrices are on their way (cp.async) and its rows of u are held in registers, split when the buffer is free.
constexpr int kGT = 64, kGC = 64, kGK = 32, kGP = kGK + 8;
struct GateTiles {
    __nv_bfloat16 u[3][kGT][kGP];
    __nv_bfloat16 w[2][kGC][kGP];
};

__global__ void __launch_bounds__(256)
lru_gates_tc_kernel(const float* __restrict__ u, const __nv_bfloat16* __restrict__ wr, const __nv_bfloat16* __restrict__ wi,
                    const float* __restrict__ br, const float* __restrict__ bi, const float* __restrict__ rate,
                    float* __restrict__ a_out, float* __restrict__ x_out, int T, int W, int n, int ctiles, int vec) {
    extern __shared__ __align__(16) unsigned char raw[];
    GateTiles* buf = reinterpret_cast<GateTiles*>(raw);             // two of them
    wait_for_earlier_kernels();
    const int t0 = blockIdx.x * kGT, part = blockIdx.y / ctiles, c0 = (blockIdx.y % ctiles) * kGC;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, wt = warp & 3, wc = warp >> 2;
    const int r0 = lane >> 2, c2 = (lane & 3) * 2;
    float acc[2][4][4];
#pragma unroll
    for (int g = 0; g < 2; ++g)
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[g][x][e] = 0.f;
    const __nv_bfloat16* w0 = wr + ((int64_t)part * n + c0) * n;
    const __nv_bfloat16* w1 = wi + ((int64_t)part * n + c0) * n;
    const float* ub = u + (int64_t)part * n;
    auto fetch_w = [&](int k0, GateTiles& b) {
        for (int idx = tid; idx < 2 * kGC * (kGK / 8); idx += 256) {
            const int i = 8 * (idx % (kGK / 8)), o = (idx / (kGK / 8)) % kGC, g = idx / (kGK / 8 * kGC);
            __nv_bfloat16* dst = &b.w[g][o][i];
            const __nv_bfloat16* src = (g ? w1 : w0) + (int64_t)o * n + k0 + i;
            if (vec && c0 + o < n && k0 + i + 8 <= n) {
                const uint32_t d = static_cast<uint32_t>(__cvta_generic_to_shared(dst));
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(d), "l"(src));
            } else {
#pragma unroll
                for (int x = 0; x < 8; ++x) dst[x] = c0 + o < n && k0 + i + x < n ? src[x] : __float2bfloat16_rn(0.f);
            }
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
    float4 held[2];                                                 // rows tid / 8 + 32 q, columns 4 (tid % 8) .. + 3
    auto fetch_u = [&](int k0) {
        const int i = k0 + 4 * (tid & 7);
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            const int t = t0 + (tid >> 3) + 32 * q;
            const float* p = ub + (int64_t)t * W + i;
            held[q] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (t < T) {
                if (vec && i + 4 <= n) held[q] = *reinterpret_cast<const float4*>(p);
                else { if (i < n) held[q].x = p[0]; if (i + 1 < n) held[q].y = p[1]; if (i + 2 < n) held[q].z = p[2]; if (i + 3 < n) held[q].w = p[3]; }
            }
        }
    };
    auto store_u = [&](GateTiles& b) {
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            float v[4] = {held[q].x, held[q].y, held[q].z, held[q].w};
#pragma unroll
            for (int s = 0; s < 3; ++s) {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
                uint2 w;
                w.x = *reinterpret_cast<const uint32_t*>(&lo);
                w.y = *reinterpret_cast<const uint32_t*>(&hi);
                *reinterpret_cast<uint2*>(&b.u[s][(tid >> 3) + 32 * q][4 * (tid & 7)]) = w;
                v[0] -= __bfloat162float(lo.x); v[1] -= __bfloat162float(lo.y);
                v[2] -= __bfloat162float(hi.x); v[3] -= __bfloat162float(hi.y);
            }
        }
    };
    fetch_u(0);
    fetch_w(0, buf[0]);
    int which = 0;
    for (int k0 = 0; k0 < n; k0 += kGK, which ^= 1) {
        GateTiles& b = buf[which];
        store_u(b);
        asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        __syncthreads();                        // this slice is complete; the other buffer has been read
        if (k0 + kGK < n) { fetch_w(k0 + kGK, buf[which ^ 1]); fetch_u(k0 + kGK); }
#pragma unroll
        for (int ks = 0; ks < kGK; ks += 16) {
            if (k0 + ks < n) {
                uint32_t a[3][4];
#pragma unroll
                for (int s = 0; s < 3; ++s) ldmatrix_x4(a[s], &b.u[s][wt * 16 + (lane & 15)][ks + (lane >> 4) * 8]);
#pragma unroll
                for (int g = 0; g < 2; ++g)
#pragma unroll
                    for (int x = 0; x < 4; x += 2) {
                        uint32_t w4[4];
                        ldmatrix_x4(w4, &b.w[g][wc * 32 + x * 8 + (lane >> 4) * 8 + (lane & 7)][ks + ((lane >> 3) & 1) * 8]);
#pragma unroll
                        for (int s = 2; s >= 0; --s) {
                            mma_bf16_16816(acc[g][x], a[s][0], a[s][1], a[s][2], a[s][3], w4[0], w4[1]);
                            mma_bf16_16816(acc[g][x + 1], a[s][0], a[s][1], a[s][2], a[s][3], w4[2], w4[3]);
                        }
                    }
            }
        }
    }
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int t = t0 + wt * 16 + r0 + (e >> 1) * 8, o = c0 + wc * 32 + x * 8 + c2;
            if (t < T && o < n) {
                const int c = part * n + o;
                const int64_t at = (int64_t)t * W + c;
                const bool two = o + 1 < n;
                float a0, x0, a1 = 0.f, x1 = 0.f;
                decay_drive(acc[0][x][e] + br[c], acc[1][x][e] + bi[c], rate[c], u[at], a0, x0);
                if (two) decay_drive(acc[0][x][e + 1] + br[c + 1], acc[1][x][e + 1] + bi[c + 1], rate[c + 1], u[at + 1], a1, x1);
                if (vec) {                      // (channels in fours: two neighbours lie on an 8-byte boundary)
                    *reinterpret_cast<float2*>(a_out + at) = make_float2(a0, a1);
                    *reinterpret_cast<float2*>(x_out + at) = make_float2(x0, x1);
                } else {
                    a_out[at] = a0; x_out[at] = x0;
                    if (two) { a_out[at + 1] = a1; x_out[at + 1] = x1; }
                }
            }
        }
}

// zr, zi [T, W]: the products before their biases; a replaces zr and the drive replaces zi.
__global__ void __launch_bounds__(256)
lru_prepare_kernel(const float* __restrict__ u, float* __restrict__ zr, float* __restrict__ zi, const float* __restrict__ br,
                   const float* __restrict__ bi, const float* __restrict__ rate, int64_t total, int W) {
    wait_for_earlier_kernels();
    const int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= total) return;
    const int c = (int)(idx % W);
    float a, x;
    decay_drive(zr[idx] + br[c], zi[idx] + bi[c], rate[c], u[idx], a, x);
    zr[idx] = a;
    zi[idx] = x;
}

// First pass over segments: the segment's whole decay and the state it reaches from zero.  Segment s of request b has
// the index q_start[b] / 64 + b + s.
__global__ void __launch_bounds__(128)
lru_segments_kernel(const float* __restrict__ a, const float* __restrict__ x, const int* __restrict__ q_start,
                    float* __restrict__ seg_a, float* __restrict__ seg_s, int W) {
    wait_for_earlier_kernels();
    const int c = blockIdx.x * 128 + threadIdx.x, b = blockIdx.z, q0 = q_start[b], n = q_start[b + 1] - q0;
    const int lo = blockIdx.y * kSeg, hi = min(n, lo + kSeg);
    if (c >= W || lo >= n) return;
    float A = 1.f, S = 0.f;
    for (int t = lo; t < hi; t += 8) {
        float av[8], xv[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            const int64_t at = (int64_t)(q0 + min(t + k, hi - 1)) * W + c;
            av[k] = a[at];
            xv[k] = x[at];
        }
#pragma unroll
        for (int k = 0; k < 8; ++k)
            if (t + k < hi) { S = av[k] * S + xv[k]; A *= av[k]; }
    }
    const int64_t at = (int64_t)(q0 / kSeg + b + blockIdx.y) * W + c;
    seg_a[at] = A;
    seg_s[at] = S;
}

// The state each segment starts from (in the place of the state it reached from zero).
__global__ void __launch_bounds__(128)
lru_chain_kernel(const float* __restrict__ seg_a, float* __restrict__ seg_s, const float* __restrict__ state,
                 int64_t stride, const int* __restrict__ q_start, const int* __restrict__ state_slot, int W) {
    wait_for_earlier_kernels();
    const int c = blockIdx.x * 128 + threadIdx.x, b = blockIdx.y, q0 = q_start[b], n = q_start[b + 1] - q0;
    if (c >= W) return;
    const int segs = (n + kSeg - 1) / kSeg;
    const int64_t first = (int64_t)(q0 / kSeg + b) * W + c;
    float S = state[(int64_t)state_slot[b] * stride + c];
    for (int s = 0; s < segs; s += 8) {
        float av[8], sv[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            const int64_t at = first + (int64_t)min(s + k, segs - 1) * W;
            av[k] = seg_a[at];
            sv[k] = seg_s[at];
        }
#pragma unroll
        for (int k = 0; k < 8; ++k)
            if (s + k < segs) { seg_s[first + (int64_t)(s + k) * W] = S; S = av[k] * S + sv[k]; }
    }
}

// The recurrence and the output: out = S gelu(y + by).  seg_s null: a request in one piece from its state; else a
// segment from its start.  The last tokens' thread writes the state.
template <typename AT>
__global__ void __launch_bounds__(128)
lru_scan_kernel(const float* __restrict__ a, const float* __restrict__ x, const float* __restrict__ y, int64_t ld_y,
                const float* __restrict__ by, const float* __restrict__ seg_s, float* __restrict__ state, int64_t stride,
                const int* __restrict__ q_start, const int* __restrict__ state_slot, AT* __restrict__ out, int W) {
    wait_for_earlier_kernels();
    const int c = blockIdx.x * 128 + threadIdx.x, b = blockIdx.z, q0 = q_start[b], n = q_start[b + 1] - q0;
    const int lo = blockIdx.y * kSeg, hi = seg_s ? min(n, lo + kSeg) : n;
    if (c >= W || lo >= n) return;
    float* st = state + (int64_t)state_slot[b] * stride + c;
    float S = seg_s ? seg_s[(int64_t)(q0 / kSeg + b + blockIdx.y) * W + c] : *st;
    const float bias = by[c];
    for (int t = lo; t < hi; t += 8) {
        float av[8], xv[8], yv[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            const int64_t r = q0 + min(t + k, hi - 1);
            av[k] = a[r * W + c];
            xv[k] = x[r * W + c];
            yv[k] = y[r * ld_y + c];
        }
#pragma unroll
        for (int k = 0; k < 8; ++k)
            if (t + k < hi) {
                S = av[k] * S + xv[k];
                out[(int64_t)(q0 + t + k) * W + c] = from_float<AT>(S * gelu_tanh_f(yv[k] + bias));
            }
    }
    if (hi == n) *st = S;
}

}  // namespace lru
}  // namespace mi

namespace mi {
namespace lru {

// One token per request: a cluster of blocks per (request, part), each with a slice of the part's channels.  Every block
// forms u of the whole part (its gates read all of it); a block moves on the convolution's state of its own channels
// after the cluster's barrier, when every block has read the old one.
struct DecodeArgs {
    const float* proj;          // [T, ld]
    int64_t ld;
    int col_x, col_y;
    const float* bx;            // bias of the convolution's input, of the convolution, of the second branch
    const float* conv;          // [W][taps]
    const float* bc;
    const float* by;
    const __nv_bfloat16* wr;
    const __nv_bfloat16* wi;
    const float* br;
    const float* bi;
    const float* rate;
    float* state;
    int64_t stride, s_off, c_off;
};

constexpr int kDecR = 2;                // requests a cluster serves together: the part's matrices are read once for both
constexpr int kDecCh = 4;               // channels of a warp of a block of 8 (slices of at most 32)

template <typename AT, bool PRE>        // PRE: parts of up to 256 channels in eights, slices of up to 32: a lane's weights fit registers
__global__ void __launch_bounds__(256)
lru_decode_kernel(DecodeArgs g, const int* __restrict__ q_start, const int* __restrict__ state_slot, AT* __restrict__ out,
                  int B, int W, int n, int cs, int taps) {
    extern __shared__ __align__(16) float dec_sm[];         // u of the part for two requests, then the gates' products
    const int np = (n + 7) / 8 * 8;
    float* us = dec_sm;                                     // [2][np]
    float* zs = us + kDecR * np;                            // [2][2][cs]
    asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
    const int part = blockIdx.y, c_lo = blockIdx.x * cs, nc = min(cs, n - c_lo);
    const int b0 = blockIdx.z * kDecR, nb = min(kDecR, B - b0);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    // the weights wait for no earlier kernel: this warp's channels (warp + 8 q) are asked for first
    uint4 pa[kDecCh], pd[kDecCh];
    if (PRE) {
#pragma unroll
        for (int q = 0; q < kDecCh; ++q) {
            const int o = warp + 8 * q, k = 8 * lane;
            pa[q] = pd[q] = make_uint4(0u, 0u, 0u, 0u);
            if (o < nc && k < n) {
                const int64_t at = ((int64_t)part * n + c_lo + o) * n + k;
                pa[q] = __ldg(reinterpret_cast<const uint4*>(g.wr + at));
                pd[q] = __ldg(reinterpret_cast<const uint4*>(g.wi + at));
            }
        }
    }
    wait_for_earlier_kernels();
    for (int idx = tid; idx < nb * np; idx += 256) {
        const int r = idx / np, i = idx - r * np, c = part * n + i;
        float u = 0.f;
        if (i < n) {
            const float* hist = g.state + (int64_t)state_slot[b0 + r] * g.stride + g.c_off + c;
            float h[kMaxTaps];
#pragma unroll
            for (int j = 0; j < kMaxTaps; ++j) h[j] = j + 1 < taps ? hist[(int64_t)j * W] : 0.f;
            const float in = g.proj[(int64_t)q_start[b0 + r] * g.ld + g.col_x + c] + g.bx[c];
            u = g.bc[c];
#pragma unroll
            for (int j = 0; j < kMaxTaps; ++j) if (j < taps) u += g.conv[c * taps + j] * (j + 1 < taps ? h[j] : in);
        }
        us[idx] = u;
    }
    __syncthreads();
    for (int q = 0, o = warp; o < nc; ++q, o += 8) {
        float zr[kDecR] = {0.f, 0.f}, zi[kDecR] = {0.f, 0.f};
        if (!PRE) {
            const int64_t wrow = ((int64_t)part * n + c_lo + o) * n;
            for (int k = lane; k < n; k += 32) {
                const float a = to_float(g.wr[wrow + k]), d = to_float(g.wi[wrow + k]);
                for (int r = 0; r < nb; ++r) { zr[r] += a * us[r * np + k]; zi[r] += d * us[r * np + k]; }
            }
        } else if (8 * lane < n) {
            uint4 a = pa[0], d = pd[0];
#pragma unroll
            for (int x = 1; x < kDecCh; ++x) if (q == x) { a = pa[x]; d = pd[x]; }
            const __nv_bfloat162* ap = reinterpret_cast<const __nv_bfloat162*>(&a);
            const __nv_bfloat162* dp = reinterpret_cast<const __nv_bfloat162*>(&d);
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float2 af = __bfloat1622float2(ap[x]), df = __bfloat1622float2(dp[x]);
#pragma unroll
                for (int r = 0; r < kDecR; ++r) {
                    if (r < nb) {
                        const float2 u2 = *reinterpret_cast<const float2*>(us + r * np + 8 * lane + 2 * x);
                        zr[r] += af.x * u2.x; zr[r] += af.y * u2.y;
                        zi[r] += df.x * u2.x; zi[r] += df.y * u2.y;
                    }
                }
            }
        }
#pragma unroll
        for (int r = 0; r < kDecR; ++r) {
            zr[r] = warp_sum(zr[r]);
            zi[r] = warp_sum(zi[r]);
            if (lane == 0) { zs[(2 * r) * cs + o] = zr[r]; zs[(2 * r + 1) * cs + o] = zi[r]; }
        }
    }
    cg::cluster_group cluster = cg::this_cluster();
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
    cluster.sync();                                         // the products are there; every block has read the convolution's state
    for (int idx = tid; idx < nb * nc; idx += 256) {
        const int r = idx / nc, o = idx - r * nc, c = part * n + c_lo + o;
        const int64_t t = q_start[b0 + r];
        const float* pr = g.proj + t * g.ld;
        float* row = g.state + (int64_t)state_slot[b0 + r] * g.stride;
        float* S = row + g.s_off + c;
        float* h = row + g.c_off + c;
        float a, x;
        decay_drive(zs[(2 * r) * cs + o] + g.br[c], zs[(2 * r + 1) * cs + o] + g.bi[c], g.rate[c], us[r * np + c_lo + o], a, x);
        const float s = a * *S + x;
        *S = s;
        out[t * W + c] = from_float<AT>(s * gelu_tanh_f(pr[g.col_y + c] + g.by[c]));
        for (int j = 0; j + 2 < taps; ++j) h[(int64_t)j * W] = h[(int64_t)(j + 1) * W];
        if (taps > 1) h[(int64_t)(taps - 2) * W] = pr[g.col_x + c] + g.bx[c];
    }
}

}  // namespace lru
}  // namespace mi

using namespace mi;

extern "C" {

static bool bad_lru(int W, int n, int B) {
    if (W < 1 || n < 1 || W % n || W / n > 65535 || B > 65535) {
        set_last_error("gated linear recurrence: %d channels in parts of %d, batch %d", W, n, B);
        return true;
    }
    return false;
}

// a, x [T, W] from u [T, W] with the gates' matrices [W/n][n][n] in bfloat16
int mi_lru_gates_tc(const float* u, const void* wr, const void* wi, const float* br, const float* bi, const float* rate,
                    float* a, float* x, int T, int W, int n, cudaStream_t stream) {
    if (T <= 0) return kOk;
    if (bad_lru(W, n, 1)) return kBadShape;
    const int ctiles = (n + lru::kGC - 1) / lru::kGC;
    if ((int64_t)(W / n) * ctiles > 65535) { set_last_error("gated linear recurrence: %d channels", W); return kBadShape; }
    const int vec = n % 8 == 0 && ((reinterpret_cast<uintptr_t>(u) | reinterpret_cast<uintptr_t>(wr) | reinterpret_cast<uintptr_t>(wi) |
                                    reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(x)) & 15) == 0;
    const size_t smem = 2 * sizeof(lru::GateTiles);
    cudaFuncSetAttribute(lru::lru_gates_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch_dependent(lru::lru_gates_tc_kernel, dim3((T + lru::kGT - 1) / lru::kGT, W / n * ctiles), dim3(256), smem, stream, u,
                     (const __nv_bfloat16*)wr, (const __nv_bfloat16*)wi, br, bi, rate, a, x, T, W, n, ctiles, vec);
    return finish_launch("lru_gates_tc");
}

int mi_lru_prepare(const float* u, float* zr, float* zi, const float* br, const float* bi, const float* rate, int T, int W,
                   cudaStream_t stream) {
    if (T <= 0) return kOk;
    if (bad_lru(W, W, 1)) return kBadShape;
    const int64_t total = (int64_t)T * W;
    launch_dependent(lru::lru_prepare_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, stream, u, zr, zi, br, bi,
                     rate, total, W);
    return finish_launch("lru_prepare");
}

int mi_lru_segment_tokens() { return lru::kSeg; }

// out [T, W] = S gelu(y + by); seg_a, seg_s: (T / 64 + B) * W floats each (segments of 64 tokens side by side), or null
// (every request in one piece).
int mi_lru_scan(const float* a, const float* x, const float* y, int ld_y, const float* by, float* seg_a, float* seg_s,
                float* state, int64_t stride, const int* q_start, const int* state_slot, void* out, int adtype, int B,
                int max_q_len, int W, cudaStream_t stream) {
    if (B <= 0 || max_q_len <= 0) return kOk;
    if (bad_lru(W, W, B)) return kBadShape;
    if ((seg_a == nullptr) != (seg_s == nullptr)) { set_last_error("gated linear recurrence: half of its scratch"); return kBadShape; }
    const int cb = (W + 127) / 128, segs = seg_a ? (max_q_len + lru::kSeg - 1) / lru::kSeg : 1;
    if (segs > 65535) { set_last_error("gated linear recurrence: a portion of %d tokens", max_q_len); return kBadShape; }
    int launched = 1;
    if (seg_a) {
        launch_dependent(lru::lru_segments_kernel, dim3(cb, segs, B), dim3(128), 0, stream, a, x, q_start, seg_a, seg_s, W);
        launch_dependent(lru::lru_chain_kernel, dim3(cb, B), dim3(128), 0, stream, (const float*)seg_a, seg_s,
                         (const float*)state, stride, q_start, state_slot, W);
        launched = 3;
    }
    MI_DISPATCH_1(adtype, AT,
        launch_dependent(lru::lru_scan_kernel<AT>, dim3(cb, segs, B), dim3(128), 0, stream, a, x, y, ld_y, by,
                         (const float*)seg_s, state, stride, q_start, state_slot, (AT*)out, W));
    return finish_launch("lru_scan", launched);
}

// One token per request (checked by the caller): convolution, gates, recurrence and output.
int mi_lru_decode(const float* proj, int ld, int col_x, int col_y, const float* bx, const float* conv, const float* bc,
                  const float* by, const void* wr, const void* wi, const float* br, const float* bi, const float* rate,
                  float* state, int64_t stride, int64_t s_off, int64_t c_off, const int* q_start, const int* state_slot,
                  void* out, int adtype, int B, int W, int n, int taps, cudaStream_t stream) {
    if (B <= 0) return kOk;
    if (bad_lru(W, n, B)) return kBadShape;
    if (taps < 1 || taps > lru::kMaxTaps) { set_last_error("gated linear recurrence: %d taps", taps); return kBadShape; }
    int slices = (n + 31) / 32;
    if (slices > 8) slices = 8;
    const int cs = (n + slices - 1) / slices;
    slices = (n + cs - 1) / cs;
    const size_t smem = sizeof(float) * (lru::kDecR * ((n + 7) / 8 * 8) + 2 * lru::kDecR * cs);
    if (smem > 200 * 1024) { set_last_error("gated linear recurrence: parts of %d channels", n); return kBadShape; }
    const bool pre = n % 8 == 0 && n <= 256 && cs <= 32 && ((reinterpret_cast<uintptr_t>(wr) | reinterpret_cast<uintptr_t>(wi)) & 15) == 0;
    const lru::DecodeArgs g = {proj, ld, col_x, col_y, bx, conv, bc, by, (const __nv_bfloat16*)wr, (const __nv_bfloat16*)wi,
                               br, bi, rate, state, stride, s_off, c_off};
    cudaLaunchConfig_t lc = {};
    lc.gridDim = dim3(slices, W / n, (B + lru::kDecR - 1) / lru::kDecR);
    lc.blockDim = dim3(256);
    lc.dynamicSmemBytes = smem;
    lc.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = slices;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    lc.attrs = attr;
    lc.numAttrs = dependent_launch_enabled() ? 2 : 1;
#define MI_LRU_DECODE(PRE)                                                                                            \
    MI_DISPATCH_1(adtype, AT, {                                                                                       \
        if (smem > 48 * 1024)                                                                                         \
            cudaFuncSetAttribute(lru::lru_decode_kernel<AT, PRE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        (void)cudaLaunchKernelEx(&lc, lru::lru_decode_kernel<AT, PRE>, g, q_start, state_slot, (AT*)out, B, W, n, cs, taps); \
    })
    if (pre) MI_LRU_DECODE(true); else MI_LRU_DECODE(false);
#undef MI_LRU_DECODE
    return finish_launch("lru_decode");
}

}  // extern "C"
