// A linear recurrence per channel with gates that are products of the channels of one part (real-gated linear recurrent
// unit):  with u the output of a short convolution over time, split into `blocks` equal parts of n channels,
//
//   r = logistic(A_b u_b + ra),  i = logistic(I_b u_b + ri)        A_b, I_b [n, n], one pair per part
//   log a = -8 r softplus(lam),  S_t = a S_(t-1) + sqrt(1 - a^2) i u,  out = S gelu(y + bias)
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
__device__ __forceinline__ float softplus_f(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// decay and drive of a channel from its gates' inputs; 1 - a^2 = -(e^(2 log a) - 1) without cancellation
__device__ __forceinline__ void decay_drive(float zr, float zi, float lam, float u, float& a, float& x) {
    const float log_a = -8.0f * sigmoid_f(zr) * softplus_f(lam);
    a = expf(log_a);
    x = sqrtf(-expm1f(2.0f * log_a)) * sigmoid_f(zi) * u;
}

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* smem_row) {
    const uint32_t addr = static_cast<uint32_t>(__cvta_generic_to_shared(smem_row));
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

// Block = 4 warps: 64 tokens x 32 output channels of one part, both gates.  ra, ri [blocks][n][n] bfloat16 (out, in).
constexpr int kGT = 64, kGC = 32, kGK = 64, kGP = kGK + 8;

__global__ void __launch_bounds__(128)
lru_gates_tc_kernel(const float* __restrict__ u, const __nv_bfloat16* __restrict__ wr, const __nv_bfloat16* __restrict__ wi,
                    const float* __restrict__ br, const float* __restrict__ bi, const float* __restrict__ lam,
                    float* __restrict__ a_out, float* __restrict__ x_out, int T, int W, int n, int ctiles) {
    __shared__ __align__(16) __nv_bfloat16 Us[3][kGT][kGP];
    __shared__ __align__(16) __nv_bfloat16 Ws[2][kGC][kGP];
    wait_for_earlier_kernels();
    const int t0 = blockIdx.x * kGT, part = blockIdx.y / ctiles, c0 = (blockIdx.y % ctiles) * kGC;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, r0 = lane >> 2, c2 = (lane & 3) * 2;
    float acc[2][4][4];
#pragma unroll
    for (int g = 0; g < 2; ++g)
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[g][x][e] = 0.f;
    const __nv_bfloat16* w0 = wr + ((int64_t)part * n + c0) * n;
    const __nv_bfloat16* w1 = wi + ((int64_t)part * n + c0) * n;
    for (int k0 = 0; k0 < n; k0 += kGK) {
        __syncthreads();
        for (int idx = tid; idx < kGT * (kGK / 2); idx += 128) {
            const int j = idx / (kGK / 2), i = 2 * (idx % (kGK / 2));
            float v[2];
#pragma unroll
            for (int x = 0; x < 2; ++x)
                v[x] = (t0 + j < T && k0 + i + x < n) ? u[(int64_t)(t0 + j) * W + part * n + k0 + i + x] : 0.f;
#pragma unroll
            for (int s = 0; s < 3; ++s) {
                __nv_bfloat162 p = __floats2bfloat162_rn(v[0], v[1]);
                *reinterpret_cast<__nv_bfloat162*>(&Us[s][j][i]) = p;
                v[0] -= __bfloat162float(p.x);
                v[1] -= __bfloat162float(p.y);
            }
        }
        for (int idx = tid; idx < 2 * kGC * kGK; idx += 128) {
            const int i = idx % kGK, o = (idx / kGK) % kGC, g = idx / (kGK * kGC);
            __nv_bfloat16 v = __float2bfloat16_rn(0.f);
            if (c0 + o < n && k0 + i < n) v = (g ? w1 : w0)[(int64_t)o * n + k0 + i];
            Ws[g][o][i] = v;
        }
        __syncthreads();
#pragma unroll
        for (int ks = 0; ks < kGK; ks += 16) {
            if (k0 + ks < n) {
                uint32_t a[3][4];
#pragma unroll
                for (int s = 0; s < 3; ++s) ldmatrix_x4(a[s], &Us[s][warp * 16 + (lane & 15)][ks + (lane >> 4) * 8]);
#pragma unroll
                for (int g = 0; g < 2; ++g)
#pragma unroll
                    for (int x = 0; x < 4; ++x) {
                        const uint32_t b0 = *reinterpret_cast<const uint32_t*>(&Ws[g][x * 8 + r0][ks + c2]);
                        const uint32_t b1 = *reinterpret_cast<const uint32_t*>(&Ws[g][x * 8 + r0][ks + 8 + c2]);
#pragma unroll
                        for (int s = 2; s >= 0; --s) mma_bf16_16816(acc[g][x], a[s][0], a[s][1], a[s][2], a[s][3], b0, b1);
                    }
            }
        }
    }
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int t = t0 + warp * 16 + r0 + (e >> 1) * 8, o = c0 + x * 8 + c2 + (e & 1);
            if (t < T && o < n) {
                const int c = part * n + o;
                float a, dr;
                decay_drive(acc[0][x][e] + br[c], acc[1][x][e] + bi[c], lam[c], u[(int64_t)t * W + c], a, dr);
                a_out[(int64_t)t * W + c] = a;
                x_out[(int64_t)t * W + c] = dr;
            }
        }
}

// zr, zi [T, W]: the products before their biases; a replaces zr and the drive replaces zi.
__global__ void __launch_bounds__(256)
lru_prepare_kernel(const float* __restrict__ u, float* __restrict__ zr, float* __restrict__ zi, const float* __restrict__ br,
                   const float* __restrict__ bi, const float* __restrict__ lam, int64_t total, int W) {
    wait_for_earlier_kernels();
    const int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= total) return;
    const int c = (int)(idx % W);
    float a, x;
    decay_drive(zr[idx] + br[c], zi[idx] + bi[c], lam[c], u[idx], a, x);
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
    const float* lam;
    float* state;
    int64_t stride, s_off, c_off;
};

template <typename AT>
__global__ void __launch_bounds__(256)
lru_decode_kernel(DecodeArgs g, const int* __restrict__ q_start, const int* __restrict__ state_slot, AT* __restrict__ out,
                  int W, int n, int cs, int taps, int vec) {
    extern __shared__ __align__(16) float us[];             // [n rounded up to 8] u of the part, [cs] its newest input
    asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
    wait_for_earlier_kernels();
    const int b = blockIdx.z, part = blockIdx.y, c_lo = blockIdx.x * cs, nc = min(cs, n - c_lo);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int64_t t = q_start[b];
    float* row = g.state + (int64_t)state_slot[b] * g.stride;
    float* hist = row + g.c_off + part * n;
    const float* pr = g.proj + t * g.ld;
    for (int i = tid; i < n; i += 256) {
        const int c = part * n + i;
        float u = g.bc[c];
        for (int j = 0; j + 1 < taps; ++j) u += g.conv[c * taps + j] * hist[(int64_t)j * W + i];
        us[i] = u + g.conv[c * taps + taps - 1] * (pr[g.col_x + c] + g.bx[c]);
    }
    for (int i = n + tid; i < (n + 7) / 8 * 8; i += 256) us[i] = 0.f;
    __syncthreads();
    for (int o = warp; o < nc; o += 8) {
        const int64_t wrow = ((int64_t)part * n + c_lo + o) * n;
        float zr = 0.f, zi = 0.f;
        if (vec) {
            for (int k = 8 * lane; k < n; k += 256) {
                const uint4 a = *reinterpret_cast<const uint4*>(g.wr + wrow + k), d = *reinterpret_cast<const uint4*>(g.wi + wrow + k);
                const __nv_bfloat162* ap = reinterpret_cast<const __nv_bfloat162*>(&a);
                const __nv_bfloat162* dp = reinterpret_cast<const __nv_bfloat162*>(&d);
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    const float2 af = __bfloat1622float2(ap[x]), df = __bfloat1622float2(dp[x]);
                    const float u0 = us[k + 2 * x], u1 = us[k + 2 * x + 1];
                    zr += af.x * u0; zr += af.y * u1;
                    zi += df.x * u0; zi += df.y * u1;
                }
            }
        } else {
            for (int k = lane; k < n; k += 32) {
                zr += to_float(g.wr[wrow + k]) * us[k];
                zi += to_float(g.wi[wrow + k]) * us[k];
            }
        }
        zr = warp_sum(zr);
        zi = warp_sum(zi);
        if (lane == 0) {
            const int c = part * n + c_lo + o;
            float a, x;
            decay_drive(zr + g.br[c], zi + g.bi[c], g.lam[c], us[c_lo + o], a, x);
            float* S = row + g.s_off + c;
            const float s = a * *S + x;
            *S = s;
            out[t * W + c] = from_float<AT>(s * gelu_tanh_f(pr[g.col_y + c] + g.by[c]));
        }
    }
    cg::cluster_group cluster = cg::this_cluster();
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
    cluster.sync();                                         // every block has read the convolution's state
    for (int i = tid; i < nc; i += 256) {
        const int c = part * n + c_lo + i;
        float* h = hist + c_lo + i;
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
int mi_lru_gates_tc(const float* u, const void* wr, const void* wi, const float* br, const float* bi, const float* lam,
                    float* a, float* x, int T, int W, int n, cudaStream_t stream) {
    if (T <= 0) return kOk;
    if (bad_lru(W, n, 1)) return kBadShape;
    const int ctiles = (n + lru::kGC - 1) / lru::kGC;
    if ((int64_t)(W / n) * ctiles > 65535) { set_last_error("gated linear recurrence: %d channels", W); return kBadShape; }
    launch_dependent(lru::lru_gates_tc_kernel, dim3((T + lru::kGT - 1) / lru::kGT, W / n * ctiles), dim3(128), 0, stream, u,
                     (const __nv_bfloat16*)wr, (const __nv_bfloat16*)wi, br, bi, lam, a, x, T, W, n, ctiles);
    return finish_launch("lru_gates_tc");
}

int mi_lru_prepare(const float* u, float* zr, float* zi, const float* br, const float* bi, const float* lam, int T, int W,
                   cudaStream_t stream) {
    if (T <= 0) return kOk;
    if (bad_lru(W, W, 1)) return kBadShape;
    const int64_t total = (int64_t)T * W;
    launch_dependent(lru::lru_prepare_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, stream, u, zr, zi, br, bi,
                     lam, total, W);
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
                  const float* by, const void* wr, const void* wi, const float* br, const float* bi, const float* lam,
                  float* state, int64_t stride, int64_t s_off, int64_t c_off, const int* q_start, const int* state_slot,
                  void* out, int adtype, int B, int W, int n, int taps, cudaStream_t stream) {
    if (B <= 0) return kOk;
    if (bad_lru(W, n, B)) return kBadShape;
    if (taps < 1 || taps > lru::kMaxTaps) { set_last_error("gated linear recurrence: %d taps", taps); return kBadShape; }
    int slices = (n + 31) / 32;
    if (slices > 8) slices = 8;
    const int cs = (n + slices - 1) / slices;
    slices = (n + cs - 1) / cs;
    const size_t smem = sizeof(float) * ((n + 7) / 8 * 8);
    if (smem > 200 * 1024) { set_last_error("gated linear recurrence: parts of %d channels", n); return kBadShape; }
    const int vec = n % 8 == 0 && ((reinterpret_cast<uintptr_t>(wr) | reinterpret_cast<uintptr_t>(wi)) & 15) == 0;
    const lru::DecodeArgs g = {proj, ld, col_x, col_y, bx, conv, bc, by, (const __nv_bfloat16*)wr, (const __nv_bfloat16*)wi,
                               br, bi, lam, state, stride, s_off, c_off};
    cudaLaunchConfig_t lc = {};
    lc.gridDim = dim3(slices, W / n, B);
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
    MI_DISPATCH_1(adtype, AT, {
        if (smem > 48 * 1024)
            cudaFuncSetAttribute(lru::lru_decode_kernel<AT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        (void)cudaLaunchKernelEx(&lc, lru::lru_decode_kernel<AT>, g, q_start, state_slot, (AT*)out, W, n, cs, taps, vec);
    });
    return finish_launch("lru_decode");
}

}  // extern "C"
