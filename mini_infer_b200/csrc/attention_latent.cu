// Row-wise kernels of attention through a latent: every token keeps ONE row [c + r] that all heads share, a
// latent of c numbers (divided by its root mean square, times a gain per dimension) from which each head's
// key and value are formed by matrices of the head, followed by r numbers of a key part that is rotated by
// position and common to all heads.  With the key matrices folded into the queries
// (q'_h = W_uk,h^T q_h, so that q_h . (W_uk,h c) = q'_h . c) the attention itself is the engine's attention
// over one shared key/value head whose keys are the cached rows and whose values are their first c numbers
// (attention_shared.cu, attention_mix.cu with a value row stride, attention_prefill_tc.cu with (query, head)
// pairs as the rows of a query tile), or over keys and values formed from the gathered latents
// (attention_prefill_tc.cu); what is left for this file:
//
//   latent_rows    (latent_store) the cached row of every new token: unit-RMS latent times gain, rotated key part;
//                  (latent_query) the rotated part of every head's query into its place behind the folded part, and
//                  the unrotated part in the activation type as the operand of the folding product; both at once
//                  when one product of the layer's input holds queries and latent
//   latent_gather  the cached rows of whole contexts, one after the other: latents [rows, c] and rotated key parts
//                  [rows, r padded to 8], the operands of keys and values formed for all heads at once
//   sigmoid_gate   out[t, h, :] = a[t, h, :] * sigmoid(g[t, h, :]), the gate on the heads' outputs
//
// The rotation pairs NEIGHBOURS: dimensions 2i and 2i + 1 turn by the angle position * inv_freq[i].  Angles,
// norms and the gate are float arithmetic in both precision paths.

#include "common.cuh"

namespace mi {

struct LatentStoreArgs {
    const float* src;           // rows of `ld` floats, latent and rotated key part from column `col0` (null: none)
    int ld, col0;
    const float* gain;
    float eps;
    const int* slot_mapping;
    void* cache;                // rows of c + r
};
// A query row has H heads of [d unrotated | r rotated] floats.  Unrotated parts go to plain + (t H + h) plain_stride,
// rotated ones to rot + (t H + h) rot_stride, each followed by zeros up to plain_pad and rot_pad numbers.
struct LatentQueryArgs {
    const float* q;             // rows of `ld` floats from column `col0` (null: none)
    int ld, col0;
    void *plain, *rot;          // plain null: not wanted
    int plain_stride, rot_stride, plain_pad, rot_pad;
};

// grid (tokens, blocks per token): the blocks of a token share its heads, the first one writes the cached row.
// `magnitude` multiplies cosines and sines.
template <typename AT>
__global__ void __launch_bounds__(256)
latent_rows_kernel(LatentStoreArgs st, LatentQueryArgs qa, const int* __restrict__ positions,
                   const float* __restrict__ inv_freq, float magnitude, int H, int d, int r, int c) {
    extern __shared__ float trig[];                 // cosines, then sines, of this token's r / 2 angles
    __shared__ float red[32];
    wait_for_earlier_kernels();
    const int t = blockIdx.x;
    const int half = r / 2;
    const float pos = (float)positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        const float ang = pos * inv_freq[i];
        trig[i] = cosf(ang) * magnitude;
        trig[half + i] = sinf(ang) * magnitude;
    }
    __syncthreads();
    if (st.src && blockIdx.y == 0) {
        const int slot = st.slot_mapping[t];
        if (slot >= 0) {                            // else a row of no request: written nowhere
            const float* row = st.src + (int64_t)t * st.ld + st.col0;
            float ss = 0.f;
            for (int i = threadIdx.x; i < c; i += blockDim.x) { const float x = row[i]; ss += x * x; }
            ss = block_sum(ss, red);
            const float inv = 1.0f / sqrtf(ss / (float)c + st.eps);
            AT* out = reinterpret_cast<AT*>(st.cache) + (int64_t)slot * (c + r);
            for (int i = threadIdx.x; i < c; i += blockDim.x) out[i] = from_float<AT>(row[i] * inv * st.gain[i]);
            for (int i = threadIdx.x; i < half; i += blockDim.x) {
                const float u = row[c + 2 * i], v = row[c + 2 * i + 1];
                out[c + 2 * i] = from_float<AT>(u * trig[i] - v * trig[half + i]);
                out[c + 2 * i + 1] = from_float<AT>(v * trig[i] + u * trig[half + i]);
            }
        }
    }
    if (!qa.q) return;
    const float* row = qa.q + (int64_t)t * qa.ld + qa.col0;
    const int per = (H + gridDim.y - 1) / gridDim.y;
    const int h_lo = blockIdx.y * per, h_hi = min(H, h_lo + per);
    const int nh = h_hi - h_lo;
    if (nh <= 0) return;
    if (qa.plain) {
        AT* plain = reinterpret_cast<AT*>(qa.plain) + ((int64_t)t * H + h_lo) * qa.plain_stride;
        const int pad = qa.plain_pad;
        if (d % 4 == 0 && pad % 4 == 0 && qa.plain_stride % 4 == 0 && (qa.ld | qa.col0 | r) % 4 == 0 &&
            ((reinterpret_cast<uintptr_t>(qa.q) | reinterpret_cast<uintptr_t>(qa.plain)) & 15) == 0) {
            const int pv = pad / 4;
            for (int idx = threadIdx.x; idx < nh * pv; idx += blockDim.x) {
                const int h = idx / pv, i = (idx - h * pv) * 4;
                float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
                if (i < d) x = *reinterpret_cast<const float4*>(row + (h_lo + h) * (d + r) + i);
                store4(plain + (int64_t)h * qa.plain_stride + i, x);
            }
        } else {
            for (int idx = threadIdx.x; idx < nh * pad; idx += blockDim.x) {
                const int h = idx / pad, i = idx - h * pad;
                plain[(int64_t)h * qa.plain_stride + i] = from_float<AT>(i < d ? row[(h_lo + h) * (d + r) + i] : 0.f);
            }
        }
    }
    AT* rot = reinterpret_cast<AT*>(qa.rot) + ((int64_t)t * H + h_lo) * qa.rot_stride;
    const int hp = (qa.rot_pad > r ? qa.rot_pad : r) / 2;
    for (int idx = threadIdx.x; idx < nh * hp; idx += blockDim.x) {
        const int h = idx / hp, i = idx - h * hp;
        float a = 0.f, b = 0.f;
        if (i < half) {
            const float* p = row + (h_lo + h) * (d + r) + d + 2 * i;
            const float u = p[0], v = p[1];
            a = u * trig[i] - v * trig[half + i];
            b = v * trig[i] + u * trig[half + i];
        }
        AT* out = rot + (int64_t)h * qa.rot_stride;
        out[2 * i] = from_float<AT>(a);
        out[2 * i + 1] = from_float<AT>(b);
    }
}

// A warp per row.  The contexts of B requests follow one another; rows beyond their sum are zeros.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, const int* __restrict__ block_table,
                     const int* __restrict__ kv_len, int B, int max_pages, int page_size,
                     __nv_bfloat16* __restrict__ lat, __nv_bfloat16* __restrict__ rot, int rows, int c, int r, int rp) {
    wait_for_earlier_kernels();
    const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= rows) return;
    int b = 0, pos = row;
    while (b < B && pos >= kv_len[b]) { pos -= kv_len[b]; ++b; }
    int page = -1;
    if (b < B) page = block_table[(int64_t)b * max_pages + pos / page_size];
    const __nv_bfloat16* src = cache + ((int64_t)(page < 0 ? 0 : page) * page_size + (page < 0 ? 0 : pos % page_size)) * (c + r);
    __nv_bfloat16* dl = lat + (int64_t)row * c;
    __nv_bfloat16* dr = rot + (int64_t)row * rp;
    if (c % 8 == 0 && r % 8 == 0) {
        const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
        for (int i = lane; i < (c + r) / 8; i += 32) {
            const uint4 v = page < 0 ? zero : *(reinterpret_cast<const uint4*>(src) + i);
            if (i * 8 < c) *(reinterpret_cast<uint4*>(dl) + i) = v;
            else *(reinterpret_cast<uint4*>(dr) + (i - c / 8)) = v;
        }
        return;
    }
    const __nv_bfloat16 zero = __float2bfloat16_rn(0.f);
    for (int i = lane; i < c; i += 32) dl[i] = page < 0 ? zero : src[i];
    for (int i = lane; i < rp; i += 32) dr[i] = page < 0 || i >= r ? zero : src[c + i];
}

// out[t, h, j] = a[h * a_head + t * a_tok + j] * sigmoid(g[t * ldg + col0 + h * e + j])
template <typename AT>
__global__ void __launch_bounds__(256)
sigmoid_gate_kernel(const AT* __restrict__ a, int64_t a_head, int64_t a_tok, const float* __restrict__ g, int ldg,
                    int col0, AT* __restrict__ out, int T, int H, int e) {
    wait_for_earlier_kernels();
    const int64_t total = (int64_t)T * H * e;
    for (int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (int64_t)gridDim.x * blockDim.x) {
        const int j = (int)(idx % e);
        const int h = (int)((idx / e) % H);
        const int64_t t = idx / ((int64_t)e * H);
        const float x = to_float(a[h * a_head + t * a_tok + j]);
        const float z = g[t * ldg + col0 + h * e + j];
        out[idx] = from_float<AT>(x / (1.0f + expf(-z)));
    }
}

// bfloat16 with e a multiple of 8 and 16-byte aligned rows: eight gated values per thread
__global__ void __launch_bounds__(256)
sigmoid_gate_bf16x8_kernel(const __nv_bfloat16* __restrict__ a, int64_t a_head, int64_t a_tok,
                           const float* __restrict__ g, int ldg, int col0, __nv_bfloat16* __restrict__ out, int T,
                           int H, int e8) {
    wait_for_earlier_kernels();
    const int64_t total = (int64_t)T * H * e8;
    for (int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (int64_t)gridDim.x * blockDim.x) {
        const int j = (int)(idx % e8) * 8;
        const int h = (int)((idx / e8) % H);
        const int64_t t = idx / ((int64_t)e8 * H);
        const uint4 av = __ldg(reinterpret_cast<const uint4*>(a + h * a_head + t * a_tok + j));
        const float4* gp = reinterpret_cast<const float4*>(g + t * ldg + col0 + h * (e8 * 8) + j);
        const float4 g0 = __ldg(gp), g1 = __ldg(gp + 1);
        const __nv_bfloat162* ap = reinterpret_cast<const __nv_bfloat162*>(&av);
        const float z[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w};
        uint4 o;
        __nv_bfloat162* op = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 x = __bfloat1622float2(ap[k]);
            op[k] = __floats2bfloat162_rn(x.x / (1.0f + expf(-z[2 * k])), x.y / (1.0f + expf(-z[2 * k + 1])));
        }
        *reinterpret_cast<uint4*>(out + idx * 8) = o;
    }
}

}  // namespace mi

using namespace mi;

extern "C" {

// `src` null: no cached rows; `q` null: no queries.  q_rot rows (t, h) are rot_stride elements apart, q_plain rows
// plain_stride (null: not wanted), each written with zeros up to rot_pad and plain_pad numbers.
int mi_latent_rows(const float* src, int ld, int col0, const float* gain, float eps, const int* slot_mapping,
                   void* cache, const float* q, int q_ld, int q_col0, void* q_plain, int plain_stride, int plain_pad,
                   void* q_rot, int rot_stride, int rot_pad, const int* positions, const float* inv_freq,
                   float magnitude, int adtype, int T, int H, int d, int r, int c, cudaStream_t stream) {
    if (T <= 0) return kOk;
    if (c < 1 || r < 0 || r % 2 || (r > 0 && !inv_freq) || (!src && !q)) {
        set_last_error("latent_rows: latent of %d and rotated part of %d", c, r);
        return kBadShape;
    }
    if (src && (col0 < 0 || col0 + c + r > ld || !gain || !slot_mapping || !cache)) {
        set_last_error("latent_rows: latent of %d and rotated part of %d at column %d of rows of %d", c, r, col0, ld);
        return kBadShape;
    }
    if (q && (H < 1 || d < 1 || q_col0 < 0 || q_col0 + H * (d + r) > q_ld || (r > 0 && !q_rot) || rot_pad % 2 ||
              rot_stride < (rot_pad > r ? rot_pad : r) || (q_plain && (plain_pad < d || plain_stride < plain_pad)))) {
        set_last_error("latent_rows: %d heads of %d + %d at column %d of rows of %d", H, d, r, q_col0, q_ld);
        return kBadShape;
    }
    const LatentStoreArgs st = {src, ld, col0, gain, eps, slot_mapping, cache};
    const LatentQueryArgs qa = {q, q_ld, q_col0, q_plain, q_rot, plain_stride, rot_stride, plain_pad, rot_pad};
    // a step of few tokens spreads a token's heads over several blocks
    int by = 1;
    if (q && T <= 32) by = H >= 16 ? 4 : (H >= 4 ? 2 : 1);
    MI_DISPATCH_1(adtype, AT,
        launch_dependent(latent_rows_kernel<AT>, dim3(T, by), dim3(256), sizeof(float) * (r > 0 ? r : 1), stream, st,
                         qa, positions, inv_freq, magnitude, H, d, r, c));
    return finish_launch("latent_rows");
}

int mi_latent_gather(const void* cache, const int* block_table, const int* kv_len, int B, int max_pages, int page_size,
                     void* lat, void* rot, int rows, int c, int r, int rp, cudaStream_t stream) {
    if (rows <= 0) return kOk;
    if (B < 1 || c < 1 || r < 0 || rp < r || max_pages < 1 || page_size < 1) {
        set_last_error("latent_gather: %d requests, rows of %d + %d", B, c, r);
        return kBadShape;
    }
    launch_dependent(latent_gather_kernel, dim3((rows + 7) / 8), dim3(256), 0, stream, (const __nv_bfloat16*)cache,
                     block_table, kv_len, B, max_pages, page_size, (__nv_bfloat16*)lat, (__nv_bfloat16*)rot, rows, c, r, rp);
    return finish_launch("latent_gather");
}

int mi_sigmoid_gate(const void* a, int64_t a_head, int64_t a_tok, const float* g, int ldg, int col0, void* out,
                    int adtype, int T, int H, int e, cudaStream_t stream) {
    if (T <= 0) return kOk;
    if (H < 1 || e < 1 || col0 < 0 || col0 + H * e > ldg) {
        set_last_error("sigmoid_gate: %d heads of %d at column %d of rows of %d", H, e, col0, ldg);
        return kBadShape;
    }
    const int64_t total = (int64_t)T * H * e;
    if (adtype == kBF16 && e % 8 == 0 && a_head % 8 == 0 && a_tok % 8 == 0 && ldg % 4 == 0 && col0 % 4 == 0 &&
        ((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(g) | reinterpret_cast<uintptr_t>(out)) & 15) == 0) {
        int64_t vblocks = (total / 8 + 255) / 256;
        if (vblocks > 148 * 16) vblocks = 148 * 16;
        launch_dependent(sigmoid_gate_bf16x8_kernel, dim3((int)vblocks), dim3(256), 0, stream,
                         (const __nv_bfloat16*)a, a_head, a_tok, g, ldg, col0, (__nv_bfloat16*)out, T, H, e / 8);
        return finish_launch("sigmoid_gate");
    }
    const int blocks = (int)((total + 255) / 256 < 65535 ? (total + 255) / 256 : 65535);
    MI_DISPATCH_1(adtype, AT,
        launch_dependent(sigmoid_gate_kernel<AT>, dim3(blocks), dim3(256), 0, stream, (const AT*)a, a_head, a_tok, g,
                         ldg, col0, (AT*)out, T, H, e));
    return finish_launch("sigmoid_gate");
}

}  // extern "C"
