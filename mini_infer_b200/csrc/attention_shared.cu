// Attention of all heads of a query over ONE shared key/value head whose values are the leading part of its key rows:
// attention through a latent with the key matrices folded into the queries (attention_latent.cu).  The rows of the
// problem are (query, head) pairs: a request with n new tokens has n * H rows q [dk], all of which read the same
// cached rows [dk], and whose values are the first c numbers of those.  Causal, with an optional window.
//
//   attn_shared_tc      bfloat16, mma.sync m16n8k16.  A block owns 16, 32 or 64 rows and a range of keys ("split");
//                       a tile of 64 keys comes to shared memory by cp.async a step ahead of its use and serves as K
//                       and as V.  Per tile: each of the 8 warps forms the scores of 8 keys for all rows; the threads
//                       of a row form its maximum, exponentials and sum; each warp adds P V to its share of the
//                       value columns.  The heads of a decoding request fill the rows of a tensor-core tile (a tile
//                       per head would hold one row of sixteen), so a decode step reads its keys once.
//                       Any c and dk that are multiples of 8 (c up to 512).
//   attn_shared_plain   any sizes and both storage types, on CUDA cores: a warp per row, a lane per key of a tile of
//                       32.  Tiles lie at absolute positions and every sum runs in an order that depends on the
//                       row's own position only: the result does not depend on how a prompt was cut.
//   latent_values       for steps of few tokens: the partial results of the splits merged, the head's value matrix
//                       applied, the output gate, one block per (token, head)
//   latent_fold         for steps of few tokens: every head's queries folded by its key matrix, their rotated parts,
//                       and the tokens' cached rows

#include "common.cuh"

namespace mi {
namespace sh {

constexpr int KT = 64;             // keys per tile

__device__ __forceinline__ void ldm_x4(uint32_t (&r)[4], const void* p) {
    const uint32_t a = static_cast<uint32_t>(__cvta_generic_to_shared(p));
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldm_x2(uint32_t& r0, uint32_t& r1, const void* p) {
    const uint32_t a = static_cast<uint32_t>(__cvta_generic_to_shared(p));
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];\n" : "=r"(r0), "=r"(r1) : "r"(a));
}
__device__ __forceinline__ void ldm_x4_trans(uint32_t (&r)[4], const void* p) {
    const uint32_t a = static_cast<uint32_t>(__cvta_generic_to_shared(p));
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void copy_16(void* smem_dst, const void* src) {
    const uint32_t dst = static_cast<uint32_t>(__cvta_generic_to_shared(smem_dst));
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(src));
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// MT: tiles of 16 rows per block.  NTW: tiles of 8 value columns per warp.
template <int MT, int NTW>
__global__ void __launch_bounds__(256)
attn_shared_tc_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ cache,
                      const int* __restrict__ block_table, const int* __restrict__ q_start,
                      const int* __restrict__ kv_len, __nv_bfloat16* __restrict__ out, float* __restrict__ part_o,
                      float* __restrict__ part_ml, int H, int dk, int c, int page_size, int max_pages, int window,
                      float scale_log2, int splits, int total_rows) {
    constexpr int BM = 16 * MT;
    constexpr int SP = KT + 4, PP = KT + 8;
    constexpr int TPR = 256 / BM, KPT = KT / TPR;          // threads of a row, keys of a thread
    extern __shared__ __align__(16) unsigned char smem_raw[];
    wait_for_earlier_kernels();
    const int b = blockIdx.y, split = blockIdx.z;
    const int q0 = q_start[b], q_len = q_start[b + 1] - q0;
    const int R = q_len * H;
    const int row0 = blockIdx.x * BM;
    if (row0 >= R) return;
    const int kvl = kv_len[b];
    const int nr = min(BM, R - row0);
    const int p_base = kvl - q_len;                        // position of the request's first query of this step
    const int p_lo = p_base + row0 / H, p_hi = p_base + (row0 + nr - 1) / H;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int dkp = (dk + 15) & ~15, pitch = dkp + 8;      // an odd number of 16-byte pieces: no bank conflicts
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);      // [BM][pitch]
    __nv_bfloat16* Ks = Qs + (size_t)BM * pitch;                         // [2][KT][pitch]
    __nv_bfloat16* Ps = Ks + (size_t)2 * KT * pitch;                     // [BM][PP]
    float* Ss = reinterpret_cast<float*>(Ps + (size_t)BM * PP);          // [BM][SP]
    float* alpha_s = Ss + BM * SP;                                       // [BM]
    float* l_s = alpha_s + BM;                                           // [BM]

    int k_begin = window > 0 ? max(0, p_lo - window + 1) / KT * KT : 0;
    const int k_limit = min(kvl, p_hi + 1);
    int n_tiles = (k_limit - k_begin + KT - 1) / KT;
    if (splits > 1) {
        const int per = (n_tiles + splits - 1) / splits;
        k_begin += split * per * KT;
        n_tiles = min(per, n_tiles - split * per);
    }
    const int* table = block_table + (size_t)b * max_pages;
    const int chunks = dk / 8, pchunks = dkp / 8;
    auto fetch = [&](int ti) {
        __nv_bfloat16* dst0 = Ks + (size_t)(ti & 1) * KT * pitch;
        const int k0 = k_begin + ti * KT;
        // a warp per key: one table entry for all lanes, 16 bytes a lane
        for (int j = warp; j < KT; j += 8) {
            const int kj = k0 + j;
            int page = -1;
            if (kj < k_limit) page = table[kj / page_size];
            __nv_bfloat16* dst = dst0 + (size_t)j * pitch;
            const __nv_bfloat16* src = cache + ((size_t)page * page_size + kj % page_size) * dk;
            for (int c8 = lane; c8 < pchunks; c8 += 32) {
                if (page >= 0 && c8 < chunks) copy_16(dst + c8 * 8, src + c8 * 8);
                else *reinterpret_cast<uint4*>(dst + c8 * 8) = make_uint4(0, 0, 0, 0);
            }
        }
    };
    if (n_tiles > 0) fetch(0);
    for (int idx = tid; idx < BM * pchunks; idx += 256) {
        const int i = idx / pchunks, c8 = idx - i * pchunks;
        __nv_bfloat16* dst = Qs + (size_t)i * pitch + c8 * 8;
        if (i < nr && c8 < chunks) copy_16(dst, q + ((size_t)q0 * H + row0 + i) * dk + c8 * 8);
        else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
    }
    copy_commit();

    float acc[MT][NTW][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < NTW; ++n)
#pragma unroll
            for (int x = 0; x < 4; ++x) acc[m][n][x] = 0.f;
    const int my_row = tid / TPR, my_key = (tid % TPR) * KPT;            // of the softmax
    const int my_pos = p_base + (row0 + my_row) / H;
    const int my_lo = window > 0 ? my_pos - window + 1 : 0;
    float m_run = -INFINITY, l_run = 0.f;                                // maximum in log2 units

    for (int ti = 0; ti < n_tiles; ++ti) {
        if (ti + 1 < n_tiles) fetch(ti + 1);
        copy_commit();
        copy_wait<1>();
        __syncthreads();
        const __nv_bfloat16* kt = Ks + (size_t)(ti & 1) * KT * pitch;
        // ---- scores: this warp's 8 keys, all rows; two chains of products per row tile ----
        {
            float s[MT][2][4];
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int x = 0; x < 4; ++x) s[m][0][x] = s[m][1][x] = 0.f;
            const __nv_bfloat16* kr = kt + (size_t)(warp * 8 + (lane & 7)) * pitch + (lane >> 3) * 8;
            const __nv_bfloat16* qr = Qs + (size_t)(lane & 15) * pitch + (lane >> 4) * 8;
            int ks = 0;
            for (; ks + 32 <= dkp; ks += 32) {
                uint32_t bf[4];
                ldm_x4(bf, kr + ks);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    uint32_t a[4];
                    ldm_x4(a, qr + (size_t)m * 16 * pitch + ks);
                    mma_bf16_16816(s[m][0], a[0], a[1], a[2], a[3], bf[0], bf[1]);
                    ldm_x4(a, qr + (size_t)m * 16 * pitch + ks + 16);
                    mma_bf16_16816(s[m][1], a[0], a[1], a[2], a[3], bf[2], bf[3]);
                }
            }
            if (ks < dkp) {
                uint32_t b0, b1;
                ldm_x2(b0, b1, kt + (size_t)(warp * 8 + (lane & 7)) * pitch + ((lane >> 3) & 1) * 8 + ks);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    uint32_t a[4];
                    ldm_x4(a, qr + (size_t)m * 16 * pitch + ks);
                    mma_bf16_16816(s[m][0], a[0], a[1], a[2], a[3], b0, b1);
                }
            }
            const int r = lane >> 2, cc = warp * 8 + (lane & 3) * 2;
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                float2* d0 = reinterpret_cast<float2*>(Ss + (m * 16 + r) * SP + cc);
                float2* d1 = reinterpret_cast<float2*>(Ss + (m * 16 + r + 8) * SP + cc);
                *d0 = make_float2(s[m][0][0] + s[m][1][0], s[m][0][1] + s[m][1][1]);
                *d1 = make_float2(s[m][0][2] + s[m][1][2], s[m][0][3] + s[m][1][3]);
            }
        }
        __syncthreads();
        // ---- softmax: TPR threads a row ----
        {
            const int k0 = k_begin + ti * KT + my_key;
            float v[KPT];
            float mx = -INFINITY;
#pragma unroll
            for (int i = 0; i < KPT; ++i) {
                const int kj = k0 + i;
                const bool vis = kj <= my_pos && kj >= my_lo && kj < k_limit;
                v[i] = vis ? Ss[my_row * SP + my_key + i] * scale_log2 : -INFINITY;
                mx = fmaxf(mx, v[i]);
            }
#pragma unroll
            for (int o = TPR / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m_run, mx);
            const float al = mn == -INFINITY ? 1.f : exp2_fast(m_run - mn);
            float sum = 0.f;
#pragma unroll
            for (int i = 0; i < KPT; ++i) {
                v[i] = mn == -INFINITY ? 0.f : exp2_fast(v[i] - mn);
                sum += v[i];
            }
#pragma unroll
            for (int i = 0; i < KPT; i += 2)
                *reinterpret_cast<uint32_t*>(Ps + my_row * PP + my_key + i) = pack2(v[i], v[i + 1]);
#pragma unroll
            for (int o = TPR / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            l_run = l_run * al + sum;
            m_run = mn;
            if (tid % TPR == 0) alpha_s[my_row] = al;
        }
        __syncthreads();
        // ---- O = O alpha + P V ----
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const float a0 = alpha_s[m * 16 + (lane >> 2)], a1 = alpha_s[m * 16 + (lane >> 2) + 8];
#pragma unroll
            for (int n = 0; n < NTW; ++n) {
                acc[m][n][0] *= a0; acc[m][n][1] *= a0;
                acc[m][n][2] *= a1; acc[m][n][3] *= a1;
            }
        }
#pragma unroll
        for (int kk = 0; kk < KT / 32; ++kk) {
            uint32_t pa[MT][2][4];
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                const __nv_bfloat16* pr = Ps + (size_t)(m * 16 + (lane & 15)) * PP + kk * 32 + (lane >> 4) * 8;
                ldm_x4(pa[m][0], pr);
                ldm_x4(pa[m][1], pr + 16);
            }
            const __nv_bfloat16* vr = kt + (size_t)(kk * 32 + lane) * pitch;
#pragma unroll
            for (int n = 0; n < NTW; ++n) {
                const int col = (warp * NTW + n) * 8;
                if (col < c) {
                    uint32_t bv[4];
                    ldm_x4_trans(bv, vr + col);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        mma_bf16_16816(acc[m][n], pa[m][0][0], pa[m][0][1], pa[m][0][2], pa[m][0][3], bv[0], bv[1]);
                        mma_bf16_16816(acc[m][n], pa[m][1][0], pa[m][1][1], pa[m][1][2], pa[m][1][3], bv[2], bv[3]);
                    }
                }
            }
        }
        __syncthreads();            // this tile's buffer and P are free for the tile after next and the next one
    }
    copy_wait<0>();                 // an empty split's query copies are still in flight
    // ---- results ----
    if (part_o) {
        if (tid % TPR == 0 && my_row < nr) {
            float* ml = part_ml + ((size_t)split * total_rows + (size_t)q0 * H + row0 + my_row) * 2;
            ml[0] = m_run;
            ml[1] = l_run;
        }
        if (n_tiles <= 0) return;   // an empty split: the merge reads its sum of 0 and nothing else
    }
    if (tid % TPR == 0) l_s[my_row] = l_run;
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m) {
        const int r = m * 16 + (lane >> 2);
#pragma unroll
        for (int n = 0; n < NTW; ++n) {
            const int col = (warp * NTW + n) * 8 + (lane & 3) * 2;
            if (col >= c) continue;
#pragma unroll
            for (int hh = 0; hh < 2; ++hh) {
                const int row = r + hh * 8;
                if (row >= nr) continue;
                const size_t grow = (size_t)q0 * H + row0 + row;
                if (part_o) {
                    *reinterpret_cast<float2*>(part_o + ((size_t)split * total_rows + grow) * c + col) =
                        make_float2(acc[m][n][hh * 2], acc[m][n][hh * 2 + 1]);
                } else {
                    const float inv = l_s[row] > 0.f ? 1.f / l_s[row] : 0.f;
                    *reinterpret_cast<uint32_t*>(out + grow * c + col) =
                        pack2(acc[m][n][hh * 2] * inv, acc[m][n][hh * 2 + 1] * inv);
                }
            }
        }
    }
}

// out[row, :] from the splits' partial results, in split order
__global__ void __launch_bounds__(128)
attn_shared_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                         __nv_bfloat16* __restrict__ out, int c, int splits, int total_rows) {
    extern __shared__ float msh[];              // [splits] weights
    wait_for_earlier_kernels();
    const size_t row = blockIdx.x;
    float m = -INFINITY;
    for (int s = 0; s < splits; ++s) m = fmaxf(m, part_ml[((size_t)s * total_rows + row) * 2]);
    float l = 0.f;
    for (int s = 0; s < splits; ++s) {
        const float ms = part_ml[((size_t)s * total_rows + row) * 2], ls = part_ml[((size_t)s * total_rows + row) * 2 + 1];
        const float w = ls > 0.f ? exp2_fast(ms - m) : 0.f;
        l += ls * w;
        if (threadIdx.x == 0) msh[s] = w;
    }
    __syncthreads();
    const float inv = l > 0.f ? 1.f / l : 0.f;
    for (int i = threadIdx.x; i < c; i += blockDim.x) {
        float o = 0.f;
        for (int s = 0; s < splits; ++s)
            if (msh[s] != 0.f) o += part_o[((size_t)s * total_rows + row) * c + i] * msh[s];
        out[row * c + i] = __float2bfloat16_rn(o * inv);
    }
}

// ---------------------------------------------------------------------------
// any sizes, CUDA cores
// ---------------------------------------------------------------------------
constexpr int PK = 32;             // keys per tile: one a lane

template <typename AT, int CPL>
__global__ void __launch_bounds__(256)
attn_shared_plain_kernel(const AT* __restrict__ q, const AT* __restrict__ cache, const int* __restrict__ block_table,
                         const int* __restrict__ q_start, const int* __restrict__ kv_len, AT* __restrict__ out, int H,
                         int dk, int c, int page_size, int max_pages, int window, float scale) {
    extern __shared__ __align__(16) float fsm[];
    wait_for_earlier_kernels();
    const int b = blockIdx.y;
    const int q0 = q_start[b], q_len = q_start[b + 1] - q0;
    const int R = q_len * H, row0 = blockIdx.x * 8;
    if (row0 >= R) return;
    const int kvl = kv_len[b];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int pitch = dk | 1;
    float* Ks = fsm;                                // [PK][pitch]
    float* Qs = Ks + PK * pitch + warp * dk;        // this warp's row
    const int row = row0 + warp;
    const bool mine = row < R;
    const int last = min(row0 + 7, R - 1);
    const int p_base = kvl - q_len;
    const int pos = p_base + (mine ? row : last) / H;
    const int p_lo = p_base + row0 / H, p_hi = p_base + last / H;
    if (mine)
        for (int i = lane; i < dk; i += 32) Qs[i] = to_float(q[((size_t)q0 * H + row) * dk + i]);
    float acc[CPL];
#pragma unroll
    for (int i = 0; i < CPL; ++i) acc[i] = 0.f;
    float m_run = -INFINITY, l_run = 0.f;
    const int k_begin = window > 0 ? max(0, p_lo - window + 1) / PK * PK : 0;
    const int k_end = min(kvl, p_hi + 1);
    const int* table = block_table + (size_t)b * max_pages;
    for (int k0 = k_begin; k0 < k_end; k0 += PK) {
        __syncthreads();
        for (int j = warp; j < PK; j += 8) {
            const int kj = k0 + j;
            int page = -1;
            if (kj < k_end) page = table[kj / page_size];
            const AT* src = cache + ((size_t)(page < 0 ? 0 : page) * page_size + kj % page_size) * dk;
            for (int i = lane; i < dk; i += 32) Ks[j * pitch + i] = page >= 0 ? to_float(src[i]) : 0.f;
        }
        __syncthreads();
        if (!mine) continue;
        const int kj = k0 + lane;
        float s = 0.f;
        const float* kr = Ks + lane * pitch;
        for (int i = 0; i < dk; ++i) s = fmaf(Qs[i], kr[i], s);
        const bool vis = kj <= pos && kj < k_end && (window == 0 || kj > pos - window);
        s = vis ? s * scale : -INFINITY;
        const float mn = fmaxf(m_run, warp_max(s));
        if (mn == -INFINITY) continue;              // uniform over the warp: nothing visible so far
        const float al = expf(m_run - mn);
        const float p = expf(s - mn);
        l_run = l_run * al + warp_sum(p);
        m_run = mn;
#pragma unroll
        for (int i = 0; i < CPL; ++i) acc[i] *= al;
        for (int j = 0; j < PK; ++j) {
            const float pj = __shfl_sync(0xffffffffu, p, j);
            const float* vr = Ks + j * pitch;
#pragma unroll
            for (int i = 0; i < CPL; ++i) {
                const int col = lane + 32 * i;
                if (col < c) acc[i] = fmaf(pj, vr[col], acc[i]);
            }
        }
    }
    if (!mine) return;
    const float inv = l_run > 0.f ? 1.f / l_run : 0.f;
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
        const int col = lane + 32 * i;
        if (col < c) out[((size_t)q0 * H + row) * c + col] = from_float<AT>(acc[i] * inv);
    }
}

// ---------------------------------------------------------------------------
// steps of few tokens: the head's matrices beside the attention
// ---------------------------------------------------------------------------

// grid (H, T).  out[t, h, :] = (W_uv,h . sum_s part) * logistic(gate) with w_uv [H, e, c] bfloat16 rows.  A warp owns e / 8
// value columns, four at a time; a lane 8 latent numbers of every 256.  The matrix does not depend on the kernels
// before: the first columns' rows are asked for before the wait.
template <int CP>                                   // passes of 256 latent numbers
__global__ void __launch_bounds__(256)
latent_values_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                     const __nv_bfloat16* __restrict__ w_uv, const float* __restrict__ gate, int ldg, int gcol,
                     __nv_bfloat16* __restrict__ out, int H, int e, int c, int splits, int total_rows) {
    extern __shared__ __align__(16) float vsm[];    // [c] merged row, [512] or more shares of it, [splits] weights
    float* share = vsm + c;
    float* wgt = share + (c > 512 ? c : 512);
    const int h = blockIdx.x, t = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int c8n = c / 8;
    const int per = (e + 7) / 8, i_lo = warp * per, i_hi = min(e, i_lo + per);
    const uint4* wrow = reinterpret_cast<const uint4*>(w_uv + (size_t)h * e * c);
    uint4 w[4][CP];
    auto fetch = [&](int i0) {
#pragma unroll
        for (int k = 0; k < 4; ++k)
#pragma unroll
            for (int p = 0; p < CP; ++p) {
                const int c8 = lane + 32 * p;
                w[k][p] = i0 + k < i_hi && c8 < c8n ? __ldg(wrow + (size_t)(i0 + k) * c8n + c8) : make_uint4(0, 0, 0, 0);
            }
    };
    fetch(i_lo);
    wait_for_earlier_kernels();
    const size_t row = (size_t)t * H + h;
    // The threads form groups that own all columns, two a thread, and every ng-th split.  The partial results are asked
    // for while the splits' weights are formed.
    const int half = c / 2, ng = 256 / half, g = threadIdx.x / half, i2 = (threadIdx.x - g * half) * 2;
    const bool mine = g < ng;
    const float2* po = reinterpret_cast<const float2*>(part_o + row * c + i2);
    const size_t step = (size_t)total_rows * half;
    constexpr int PF = 8;
    float2 pv[PF];
#pragma unroll
    for (int j = 0; j < PF; ++j) {
        const int s = g + j * ng;
        pv[j] = mine && s < splits ? __ldg(po + s * step) : make_float2(0.f, 0.f);
    }
    if (warp == 0) {
        float m = -INFINITY;
        for (int s = lane; s < splits; s += 32) m = fmaxf(m, part_ml[((size_t)s * total_rows + row) * 2]);
        m = warp_max(m);
        float l = 0.f;
        for (int s = lane; s < splits; s += 32) {
            const float2 ml = *reinterpret_cast<const float2*>(part_ml + ((size_t)s * total_rows + row) * 2);
            const float x = ml.y > 0.f ? exp2_fast(ml.x - m) : 0.f;
            wgt[s] = x;
            l += ml.y * x;
        }
        l = warp_sum(l);
        const float inv = l > 0.f ? 1.f / l : 0.f;
        for (int s = lane; s < splits; s += 32) wgt[s] *= inv;
    }
    __syncthreads();
    if (mine) {
        float2 o = make_float2(0.f, 0.f);
#pragma unroll
        for (int j = 0; j < PF; ++j) {
            const int s = g + j * ng;
            const float x = s < splits ? wgt[s] : 0.f;
            if (x != 0.f) { o.x += pv[j].x * x; o.y += pv[j].y * x; }      // an empty split wrote nothing
        }
#pragma unroll 4
        for (int s = g + PF * ng; s < splits; s += ng) {
            const float x = wgt[s];
            const float2 v = x != 0.f ? __ldg(po + s * step) : make_float2(0.f, 0.f);
            o.x += v.x * x;
            o.y += v.y * x;
        }
        *reinterpret_cast<float2*>((ng > 1 ? share + (size_t)g * c : vsm) + i2) = o;
    }
    __syncthreads();
    if (ng > 1) {
        for (int i = threadIdx.x; i < c; i += 256) {
            float o = 0.f;
            for (int k = 0; k < ng; ++k) o += share[(size_t)k * c + i];
            vsm[i] = o;
        }
        __syncthreads();
    }
    for (int i0 = i_lo; i0 < i_hi; i0 += 4) {
        float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int p = 0; p < CP; ++p) {
            const int c8 = lane + 32 * p;
            if (c8 < c8n) {
                const float4 a = *reinterpret_cast<const float4*>(vsm + c8 * 8), bq = *reinterpret_cast<const float4*>(vsm + c8 * 8 + 4);
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const __nv_bfloat162* x = reinterpret_cast<const __nv_bfloat162*>(&w[k][p]);
                    const float2 x0 = __bfloat1622float2(x[0]), x1 = __bfloat1622float2(x[1]),
                                 x2 = __bfloat1622float2(x[2]), x3 = __bfloat1622float2(x[3]);
                    s[k] += a.x * x0.x + a.y * x0.y + a.z * x1.x + a.w * x1.y + bq.x * x2.x + bq.y * x2.y + bq.z * x3.x + bq.w * x3.y;
                }
            }
        }
        if (i0 + 4 < i_hi) fetch(i0 + 4);           // the next columns' rows fly during the sums over the lanes
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float v = warp_sum(s[k]);
            if (lane == 0 && i0 + k < i_hi) {
                float o = v;
                if (gate) o = v / (1.0f + expf(-gate[(size_t)t * ldg + gcol + h * e + i0 + k]));
                out[row * e + i0 + k] = __float2bfloat16_rn(o);
            }
        }
    }
}

// grid (H, ceil(c / 32)), all tokens (at most TT) at once: q_full[t, h] = [W_uk,h^T q_plain | rot(q_rot)] with w_uk
// [H, d, c] bfloat16 read once.  A block owns 32 latent columns of one head: a thread 8 of them and every 64th query
// dimension.  The first block of a head rotates its queries; the tokens' cached rows (src null: none) are shared out
// over all blocks.  Query rows: [d | r] floats per head from column q_col.
constexpr int kFoldCols = 32;
template <int TT>
__global__ void __launch_bounds__(256)
latent_fold_kernel(const float* __restrict__ q, int q_ld, int q_col, const __nv_bfloat16* __restrict__ w_uk,
                   const float* __restrict__ src, int ld, int col0, const float* __restrict__ gain, float eps,
                   const int* __restrict__ slot_mapping, __nv_bfloat16* __restrict__ cache,
                   const int* __restrict__ positions, const float* __restrict__ inv_freq, float magnitude,
                   __nv_bfloat16* __restrict__ q_full, int T, int H, int d, int r, int c) {
    extern __shared__ __align__(16) float fs[];     // [T][d] queries
    __shared__ float part[8][TT][kFoldCols];
    __shared__ float red[32];
    const int h = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int col = blockIdx.y * kFoldCols + (lane & 3) * 8, g = warp * 8 + (lane >> 2);
    const bool mine = col < c;
    const __nv_bfloat16* w = w_uk + (size_t)h * d * c + col;
    uint4 first = make_uint4(0, 0, 0, 0);           // the matrix does not depend on the kernels before
    if (mine && g < d) first = __ldg(reinterpret_cast<const uint4*>(w + (size_t)g * c));
    wait_for_earlier_kernels();
    for (int i = threadIdx.x; i < T * d; i += 256) {
        const int t = i / d;
        fs[i] = q[(size_t)t * q_ld + q_col + (size_t)h * (d + r) + (i - t * d)];
    }
    if (blockIdx.y == 0) {
        const int half = r / 2;
        for (int idx = threadIdx.x; idx < T * half; idx += 256) {
            const int t = idx / half, i = idx - t * half;
            const float ang = (float)positions[t] * inv_freq[i];
            const float cs = cosf(ang) * magnitude, sn = sinf(ang) * magnitude;
            const float* row = q + (size_t)t * q_ld + q_col + (size_t)h * (d + r) + d;
            const float u = row[2 * i], v = row[2 * i + 1];
            __nv_bfloat16* out = q_full + ((size_t)t * H + h) * (c + r) + c;
            out[2 * i] = __float2bfloat16_rn(u * cs - v * sn);
            out[2 * i + 1] = __float2bfloat16_rn(v * cs + u * sn);
        }
    }
    if (src) {
        // from the last block down: the first block of a head has its rotations to do
        const int nb = gridDim.x * gridDim.y, bid = nb - 1 - (blockIdx.y * gridDim.x + blockIdx.x);
        for (int t = bid; t < T; t += nb) {
            const int slot = slot_mapping[t];
            if (slot < 0) continue;
            const float* kr = src + (size_t)t * ld + col0;
            float ss = 0.f;
            for (int i = threadIdx.x; i < c; i += 256) { const float x = kr[i]; ss += x * x; }
            ss = block_sum(ss, red);
            const float inv = 1.0f / sqrtf(ss / (float)c + eps);
            const float pos = (float)positions[t];
            __nv_bfloat16* dst = cache + (size_t)slot * (c + r);
            for (int i = threadIdx.x; i < c; i += 256) dst[i] = __float2bfloat16_rn(kr[i] * inv * gain[i]);
            for (int i = threadIdx.x; i < r / 2; i += 256) {
                const float ang = pos * inv_freq[i];
                const float cs = cosf(ang) * magnitude, sn = sinf(ang) * magnitude;
                const float u = kr[c + 2 * i], v = kr[c + 2 * i + 1];
                dst[c + 2 * i] = __float2bfloat16_rn(u * cs - v * sn);
                dst[c + 2 * i + 1] = __float2bfloat16_rn(v * cs + u * sn);
            }
        }
    }
    __syncthreads();
    float acc[TT][8];
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
        for (int k = 0; k < 8; ++k) acc[t][k] = 0.f;
    if (mine) {
        uint4 v = first;
        for (int i = g; i < d; i += 64) {
            const uint4 now = v;
            if (i + 64 < d) v = __ldg(reinterpret_cast<const uint4*>(w + (size_t)(i + 64) * c));
            const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&now);
            float f[8];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 x = __bfloat1622float2(p[k]);
                f[2 * k] = x.x;
                f[2 * k + 1] = x.y;
            }
#pragma unroll
            for (int t = 0; t < TT; ++t)
                if (t < T) {
                    const float x = fs[t * d + i];
#pragma unroll
                    for (int k = 0; k < 8; ++k) acc[t][k] += x * f[k];
                }
        }
    }
    // the 8 lanes of a warp that share columns, then the warps
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
        for (int k = 0; k < 8; ++k) {
#pragma unroll
            for (int o = 4; o < 32; o <<= 1) acc[t][k] += __shfl_xor_sync(0xffffffffu, acc[t][k], o);
        }
    if (lane < 4)
#pragma unroll
        for (int t = 0; t < TT; ++t)
#pragma unroll
            for (int k = 0; k < 8; ++k) part[warp][t][lane * 8 + k] = acc[t][k];
    __syncthreads();
    for (int idx = threadIdx.x; idx < T * kFoldCols; idx += 256) {
        const int t = idx / kFoldCols, i = idx - t * kFoldCols, cc = blockIdx.y * kFoldCols + i;
        if (cc >= c) continue;
        float s = 0.f;
#pragma unroll
        for (int x = 0; x < 8; ++x) s += part[x][t][i];
        q_full[((size_t)t * H + h) * (c + r) + cc] = __float2bfloat16_rn(s);
    }
}

static size_t tc_smem(int mt, int dk) {
    const int bm = 16 * mt, pitch = ((dk + 15) & ~15) + 8;
    return (size_t)(bm + 2 * KT) * pitch * 2 + (size_t)bm * (KT + 8) * 2 + (size_t)bm * (KT + 4) * 4 + (size_t)2 * bm * 4;
}
// row tiles of 16 per block for a step whose longest request has `rows` rows (0: the sizes are not taken)
static int tc_tiles(int rows, int dk, int c) {
    if (c < 8 || c > 512 || c % 8 || dk % 8 || dk < c) return 0;
    int mt = rows <= 16 ? 1 : (rows <= 32 ? 2 : 4);
    while (mt > 1 && tc_smem(mt, dk) > 220 * 1024) mt /= 2;
    return tc_smem(mt, dk) <= 220 * 1024 ? mt : 0;
}
static size_t plain_smem(int dk) { return sizeof(float) * ((size_t)PK * (dk | 1) + (size_t)8 * dk); }

}  // namespace sh
}  // namespace mi

using namespace mi;

extern "C" {

int mi_attn_shared_tc_supported(int dk, int c) { return sh::tc_tiles(16, dk, c) > 0; }
int mi_attn_shared_plain_supported(int dk, int c) { return c >= 1 && c <= 1024 && dk >= c && sh::plain_smem(dk) <= 220 * 1024; }
// rows of a block of the tensor-core form in a step whose longest request has `rows` rows
int mi_attn_shared_tc_block_rows(int rows, int dk, int c) { return 16 * sh::tc_tiles(rows, dk, c); }

// q [T * H, dk], out [T * H, c] bfloat16.  part_o [splits, T * H, c] and part_ml [splits, T * H, 2] float: given, the
// unnormalised result of every split is written there; `out` null: and nothing more (latent_values reads it), else
// the splits are merged into it.
int mi_attn_shared_tc(const void* q, const void* cache, const int* block_table, const int* q_start, const int* kv_len,
                      void* out, float* part_o, float* part_ml, int T, int B, int max_q_len, int H, int dk, int c,
                      int page_size, int max_pages, int window, float scale, int splits, cudaStream_t stream) {
    if (B <= 0 || max_q_len <= 0 || T <= 0) return kOk;
    const int64_t rows = (int64_t)max_q_len * H;
    const int mt = rows > 0 && rows < (1 << 30) ? sh::tc_tiles((int)rows, dk, c) : 0;
    if (!mt || H < 1 || window < 0 || !(scale > 0.f)) {
        set_last_error("attention over a shared head: %d heads, rows of %d, values of %d are not taken", H, dk, c);
        return kBadShape;
    }
    if (splits < 1 || splits > 4096 || B > 65535 || ((splits > 1 || !out) && (!part_o || !part_ml))) {
        set_last_error("attention over a shared head: %d splits, batch %d", splits, B);
        return kBadShape;
    }
    if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(out) |
         reinterpret_cast<uintptr_t>(part_o)) & 15) {
        set_last_error("attention over a shared head: operands must be 16-byte aligned");
        return kBadShape;
    }
    const dim3 grid((unsigned)((rows + 16 * mt - 1) / (16 * mt)), B, splits);
    const size_t smem = sh::tc_smem(mt, dk);
    const float scale_log2 = scale * 1.4426950408889634f;
    float* po = splits > 1 || !out ? part_o : nullptr;
#define MI_SH(MM, NN)                                                                                              \
    do {                                                                                                           \
        auto kern = sh::attn_shared_tc_kernel<MM, NN>;                                                             \
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                        \
        launch_dependent(kern, grid, dim3(256), smem, stream, (const __nv_bfloat16*)q, (const __nv_bfloat16*)cache, \
                         block_table, q_start, kv_len, (__nv_bfloat16*)out, po, part_ml, H, dk, c, page_size,      \
                         max_pages, window, scale_log2, splits, T * H);                                            \
    } while (0)
#define MI_SHM(NN) do { if (mt == 1) MI_SH(1, NN); else if (mt == 2) MI_SH(2, NN); else MI_SH(4, NN); } while (0)
    const int ntw = (c + 63) / 64;
    if (ntw <= 1) MI_SHM(1);
    else if (ntw <= 2) MI_SHM(2);
    else if (ntw <= 4) MI_SHM(4);
    else MI_SHM(8);
#undef MI_SHM
#undef MI_SH
    int launched = 1;
    if (po && out) {
        launch_dependent(sh::attn_shared_merge_kernel, dim3(T * H), dim3(128), sizeof(float) * splits, stream,
                         (const float*)po, (const float*)part_ml, (__nv_bfloat16*)out, c, splits, T * H);
        launched = 2;
    }
    return finish_launch("attn_shared_tc", launched);
}

int mi_attn_shared_plain(const void* q, const void* cache, int adtype, const int* block_table, const int* q_start,
                         const int* kv_len, void* out, int B, int max_q_len, int H, int dk, int c, int page_size,
                         int max_pages, int window, float scale, cudaStream_t stream) {
    if (B <= 0 || max_q_len <= 0) return kOk;
    if (!mi_attn_shared_plain_supported(dk, c) || H < 1 || B > 65535 || window < 0) {
        set_last_error("attention over a shared head: %d heads, rows of %d, values of %d are not taken", H, dk, c);
        return kBadShape;
    }
    const dim3 grid((unsigned)(((int64_t)max_q_len * H + 7) / 8), B);
    const size_t smem = sh::plain_smem(dk);
    const int cpl = (c + 31) / 32;
#define MI_SHP(CC)                                                                                                 \
    MI_DISPATCH_1(adtype, AT, {                                                                                    \
        cudaFuncSetAttribute(sh::attn_shared_plain_kernel<AT, CC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        launch_dependent(sh::attn_shared_plain_kernel<AT, CC>, grid, dim3(256), smem, stream, (const AT*)q,        \
                         (const AT*)cache, block_table, q_start, kv_len, (AT*)out, H, dk, c, page_size, max_pages, \
                         window, scale);                                                                           \
    })
    if (cpl <= 4) MI_SHP(4);
    else if (cpl <= 8) MI_SHP(8);
    else if (cpl <= 16) MI_SHP(16);
    else MI_SHP(32);
#undef MI_SHP
    return finish_launch("attn_shared_plain");
}

// out [T, H, e] bfloat16; `gate` null: no gate
int mi_latent_values(const float* part_o, const float* part_ml, const void* w_uv, const float* gate, int ldg, int gcol,
                     void* out, int T, int H, int e, int c, int splits, int total_rows, cudaStream_t stream) {
    if (T <= 0) return kOk;
    if (c % 8 || c < 8 || c > 512 || e < 1 || H < 1 || splits < 1 || T > 65535 || total_rows < T * H ||
        (gate && (gcol < 0 || gcol + H * e > ldg)) || (2 * c + 512 + splits) * sizeof(float) > 48 * 1024) {
        set_last_error("latent_values: %d heads of %d values from latents of %d, %d splits", H, e, c, splits);
        return kBadShape;
    }
#define MI_LV(CP)                                                                                                  \
    launch_dependent(sh::latent_values_kernel<CP>, dim3(H, T), dim3(256), sizeof(float) * (c + 512 + splits), stream, part_o, \
                     part_ml, (const __nv_bfloat16*)w_uv, gate, ldg, gcol, (__nv_bfloat16*)out, H, e, c, splits,   \
                     total_rows)
    if (c <= 256) MI_LV(1);
    else MI_LV(2);
#undef MI_LV
    return finish_launch("latent_values");
}

int mi_latent_fold_max_tokens() { return 16; }

int mi_latent_fold(const float* q, int q_ld, int q_col, const void* w_uk, const float* src, int ld, int col0,
                   const float* gain, float eps, const int* slot_mapping, void* cache, const int* positions,
                   const float* inv_freq, float magnitude, void* q_full, int T, int H, int d, int r, int c,
                   cudaStream_t stream) {
    if (T <= 0) return kOk;
    if (c % 8 || c < 8 || c > 512 || d < 1 || H < 1 || r < 0 || r % 2 || (r > 0 && !inv_freq) || T > 65535 || q_col < 0 ||
        q_col + H * (d + r) > q_ld || (src && (col0 < 0 || col0 + c + r > ld || !gain || !slot_mapping || !cache))) {
        set_last_error("latent_fold: %d heads of %d + %d over latents of %d", H, d, r, c);
        return kBadShape;
    }
    const size_t smem = sizeof(float) * (size_t)T * d;
    if (smem > 24 * 1024 || T > mi_latent_fold_max_tokens()) {
        set_last_error("latent_fold: %d tokens, heads of %d", T, d);
        return kBadShape;
    }
#define MI_LF(TT)                                                                                                  \
    launch_dependent(sh::latent_fold_kernel<TT>, dim3(H, (c + sh::kFoldCols - 1) / sh::kFoldCols), dim3(256), smem, \
                     stream, q, q_ld, q_col, (const __nv_bfloat16*)w_uk, src, ld, col0, gain, eps, slot_mapping,   \
                     (__nv_bfloat16*)cache, positions, inv_freq, magnitude, (__nv_bfloat16*)q_full, T, H, d, r, c)
    if (T <= 4) MI_LF(4);
    else if (T <= 8) MI_LF(8);
    else MI_LF(16);
#undef MI_LF
    return finish_launch("latent_fold");
}

}  // extern "C"
