// Row-wise kernels of a residual that is kept as S parallel streams per token, x [T, S, H] in float.
//
//   streams_embed   the first streams of every token: embedding row times a constant, plus (optional) a row of a
//                   second table chosen by a hash of the token and the token before it, RMS norm (optional),
//                   written S times.  The token before a portion's first one is read from the request's paged
//                   token ids, into which the kernel writes the ids of this step.
//   streams_read    one sublayer's boundary: the update that the sublayer before left,
//                       x_t <- sum_s mix[s, t] x_s + w_out[t] y      (all streams at once from the old ones),
//                   then what the next sublayer reads, RMS norm of u = sum_t w_in[t] x_t.  With `rows` only those
//                   rows are formed and the streams are left as they are (a model's last norm).
//   relu_glu        out = max(gate, 0) * up
//
// Everything here is float arithmetic; only the outputs that feed matrix products are rounded.  A row's sums run
// in an order that depends on S and H only.

#include "common.cuh"

namespace mi {

constexpr int kMaxStreams = 32;

// ---------------------------------------------------------------------------
// embedding
// ---------------------------------------------------------------------------
struct BigramArgs {
    const void* table;              // [buckets + 1, H] (null: no second table)
    long long buckets, mul_prev, mul_cur;
    int* token_ids;                 // one layer of the paged ids: [pages, page_size]
    const int* block_table;         // [B, max_pages]
    const int* slot_mapping;        // [T]
    int max_pages, page_size;
};

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}

template <typename WT, typename NT, int V>          // V columns per access: 4 or 1
__global__ void __launch_bounds__(256)
streams_embed_kernel(const int* __restrict__ ids, const int* __restrict__ positions,
                     const int* __restrict__ req_of_token, const WT* __restrict__ table, float scale, BigramArgs bg,
                     const NT* __restrict__ weight, float eps, float* __restrict__ out, int H, int vocab, int S) {
    __shared__ float scratch[32];
    wait_for_earlier_kernels();
    const int t = blockIdx.x;
    int id = ids[t];
    // ids are validated on the host; clamp so that a bad id can never read outside the table
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    const WT* row = table + (int64_t)id * H;
    const WT* row2 = nullptr;
    if (bg.table) {
        const int pos = positions[t];
        long long at = bg.buckets;                  // a sequence's first token: the last row
        if (pos > 0) {
            long long prev = 0;
            const int b = req_of_token[t];
            if (t > 0 && req_of_token[t - 1] == b) {
                prev = ids[t - 1];
            } else {
                const int page = bg.block_table[(int64_t)b * bg.max_pages + (pos - 1) / bg.page_size];
                if (page >= 0) prev = bg.token_ids[(int64_t)page * bg.page_size + (pos - 1) % bg.page_size];
            }
            at = (prev * bg.mul_prev + (long long)id * bg.mul_cur) % bg.buckets;
        }
        row2 = reinterpret_cast<const WT*>(bg.table) + at * H;
        // the slots written here belong to this step's tokens; the one read above to a token of an earlier step
        if (threadIdx.x == 0 && bg.slot_mapping[t] >= 0) bg.token_ids[bg.slot_mapping[t]] = ids[t];
    }
    float* dst = out + (int64_t)t * S * H;
    auto value = [&](int c, float (&v)[V]) {
        if constexpr (V == 4) {
            const float4 a = load4(row + c);
            v[0] = a.x * scale; v[1] = a.y * scale; v[2] = a.z * scale; v[3] = a.w * scale;
            if (row2) {
                const float4 b = load4(row2 + c);
                v[0] += b.x; v[1] += b.y; v[2] += b.z; v[3] += b.w;
            }
        } else {
            v[0] = to_float(row[c]) * scale;
            if (row2) v[0] += to_float(row2[c]);
        }
    };
    float rr = 1.f;
    if (weight) {
        float ss = 0.f;
        for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
            float v[V];
            value(c, v);
#pragma unroll
            for (int k = 0; k < V; ++k) ss += v[k] * v[k];
        }
        ss = block_sum(ss, scratch);
        rr = 1.0f / sqrtf(ss / (float)H + eps);
    }
    for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
        float v[V];
        value(c, v);
        if (weight)
#pragma unroll
            for (int k = 0; k < V; ++k) v[k] = v[k] * rr * to_float(weight[c + k]);
        for (int s = 0; s < S; ++s) {
            if constexpr (V == 4) *reinterpret_cast<float4*>(dst + (int64_t)s * H + c) = make_float4(v[0], v[1], v[2], v[3]);
            else dst[(int64_t)s * H + c] = v[0];
        }
    }
}

// ---------------------------------------------------------------------------
// the boundary between two sublayers
// ---------------------------------------------------------------------------
// Any S and H: a column of all streams per thread, the row of u in shared memory.
template <typename AT, typename WT>
__global__ void __launch_bounds__(256)
streams_read_any_kernel(float* __restrict__ xs, const float* __restrict__ y, const float* __restrict__ mix,
                        const float* __restrict__ w_out, const float* __restrict__ w_in, const int* __restrict__ rows,
                        const WT* __restrict__ weight, AT* __restrict__ out, int S, int H, float eps) {
    extern __shared__ float urow[];                 // [H]
    __shared__ float scratch[32];
    wait_for_earlier_kernels();
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    float* x = xs + (int64_t)src * S * H;
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        float old[kMaxStreams];
        float u = 0.f;
        for (int s = 0; s < S; ++s) old[s] = x[(int64_t)s * H + c];
        if (y) {
            const float yv = y[(int64_t)src * H + c];
            for (int t = 0; t < S; ++t) {
                float v = 0.f;
                for (int s = 0; s < S; ++s) v += mix[s * S + t] * old[s];
                v += w_out[t] * yv;
                if (!rows) x[(int64_t)t * H + c] = v;
                u += w_in[t] * v;
            }
        } else {
            for (int t = 0; t < S; ++t) u += w_in[t] * old[t];
        }
        urow[c] = u;
        ss += u * u;
    }
    ss = block_sum(ss, scratch);
    const float rr = 1.0f / sqrtf(ss / (float)H + eps);
    for (int c = threadIdx.x; c < H; c += blockDim.x)
        out[(int64_t)r * H + c] = from_float<AT>(urow[c] * rr * to_float(weight[c]));
}

// S streams of rows of H = 4 * 256 * VPT floats at most, 16 bytes an access, u in registers.
template <typename AT, typename WT, int S, int VPT>
__global__ void __launch_bounds__(256)
streams_read_vec_kernel(float* __restrict__ xs, const float* __restrict__ y, const float* __restrict__ mix,
                        const float* __restrict__ w_out, const float* __restrict__ w_in, const int* __restrict__ rows,
                        const WT* __restrict__ weight, AT* __restrict__ out, int H, float eps) {
    __shared__ float scratch[32];
    wait_for_earlier_kernels();
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    const int nv = H >> 2;
    float4* x = reinterpret_cast<float4*>(xs + (int64_t)src * S * H);
    const float4* yv = y ? reinterpret_cast<const float4*>(y + (int64_t)src * H) : nullptr;
    float m[S][S], wo[S], wi[S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
        wi[s] = __ldg(w_in + s);
        wo[s] = y ? __ldg(w_out + s) : 0.f;
#pragma unroll
        for (int t = 0; t < S; ++t) m[s][t] = y ? __ldg(mix + s * S + t) : 0.f;
    }
    float4 old[VPT][S], dy[VPT], u[VPT];
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int i = threadIdx.x + 256 * j;
        dy[j] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int s = 0; s < S; ++s) old[j][s] = i < nv ? x[(int64_t)s * nv + i] : make_float4(0.f, 0.f, 0.f, 0.f);
        if (yv && i < nv) dy[j] = __ldg(yv + i);
    }
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int i = threadIdx.x + 256 * j;
        u[j] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int t = 0; t < S; ++t) {
            float4 v = old[j][t];
            if (y) {
                v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int s = 0; s < S; ++s) {
                    v.x += m[s][t] * old[j][s].x; v.y += m[s][t] * old[j][s].y;
                    v.z += m[s][t] * old[j][s].z; v.w += m[s][t] * old[j][s].w;
                }
                v.x += wo[t] * dy[j].x; v.y += wo[t] * dy[j].y; v.z += wo[t] * dy[j].z; v.w += wo[t] * dy[j].w;
                if (!rows && i < nv) x[(int64_t)t * nv + i] = v;
            }
            u[j].x += wi[t] * v.x; u[j].y += wi[t] * v.y; u[j].z += wi[t] * v.z; u[j].w += wi[t] * v.w;
        }
        ss += u[j].x * u[j].x;
        ss += u[j].y * u[j].y;
        ss += u[j].z * u[j].z;
        ss += u[j].w * u[j].w;
    }
    ss = block_sum(ss, scratch);
    const float rr = 1.0f / sqrtf(ss / (float)H + eps);
    AT* o = out + (int64_t)r * H;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int i = threadIdx.x + 256 * j;
        if (i < nv) {
            const float4 w = load4(weight + 4 * i);
            store4(o + 4 * i, make_float4(u[j].x * rr * w.x, u[j].y * rr * w.y, u[j].z * rr * w.z, u[j].w * rr * w.w));
        }
    }
}

// the residual itself, x_1 + .. + x_S after the pending update (what a reader between two layers sees)
__global__ void __launch_bounds__(256)
streams_sum_kernel(const float* __restrict__ xs, const float* __restrict__ y, const float* __restrict__ mix,
                   const float* __restrict__ w_out, float* __restrict__ out, int S, int H) {
    wait_for_earlier_kernels();
    const int r = blockIdx.x;
    const float* x = xs + (int64_t)r * S * H;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        float u = 0.f;
        for (int t = 0; t < S; ++t) {
            float v = 0.f;
            if (y) {
                for (int s = 0; s < S; ++s) v += mix[s * S + t] * x[(int64_t)s * H + c];
                v += w_out[t] * y[(int64_t)r * H + c];
            } else {
                v = x[(int64_t)t * H + c];
            }
            u += v;
        }
        out[(int64_t)r * H + c] = u;
    }
}

// ---------------------------------------------------------------------------
// gated unit with a rectified gate
// ---------------------------------------------------------------------------
template <typename AT>
__global__ void relu_glu_kernel(const AT* __restrict__ gu, AT* __restrict__ out, int64_t total, int I) {
    wait_for_earlier_kernels();
    for (int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
         idx += (int64_t)gridDim.x * blockDim.x) {
        const int64_t t = idx / I;
        const int i = (int)(idx - t * I);
        out[idx] = from_float<AT>(fmaxf(to_float(gu[t * 2 * I + i]), 0.f) * to_float(gu[t * 2 * I + I + i]));
    }
}

// bfloat16 rows with I a multiple of 8: 16 bytes per load and store
__global__ void relu_glu_bf16x8_kernel(const uint4* __restrict__ gu, uint4* __restrict__ out, int64_t total_vec,
                                       int Iv) {
    wait_for_earlier_kernels();
    for (int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total_vec;
         idx += (int64_t)gridDim.x * blockDim.x) {
        const int64_t t = idx / Iv;
        const int i = (int)(idx - t * Iv);
        const uint4 gv = __ldg(gu + t * 2 * Iv + i);
        const uint4 uv = __ldg(gu + t * 2 * Iv + Iv + i);
        const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&gv);
        const __nv_bfloat162* u2 = reinterpret_cast<const __nv_bfloat162*>(&uv);
        uint4 r;
        __nv_bfloat162* r2 = reinterpret_cast<__nv_bfloat162*>(&r);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 g = __bfloat1622float2(g2[j]), u = __bfloat1622float2(u2[j]);
            r2[j] = __floats2bfloat162_rn(fmaxf(g.x, 0.f) * u.x, fmaxf(g.y, 0.f) * u.y);
        }
        out[idx] = r;
    }
}

}  // namespace mi

using namespace mi;

static bool aligned16(const void* a, const void* b = nullptr, const void* c = nullptr, const void* d = nullptr) {
    return ((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(c) |
             reinterpret_cast<uintptr_t>(d)) & 15) == 0;
}

extern "C" {

// out [T, S, H] float.  `bigram` null: no second table (and the arguments after it are not read); `weight` null: no
// norm.  wdtype is the type of both tables, ndtype that of the norm's weight.
int mi_streams_embed(const int* ids, const int* positions, const int* req_of_token, const void* table, int wdtype,
                     float scale, const void* bigram, int64_t buckets, int64_t mul_prev, int64_t mul_cur,
                     int* token_ids, const int* block_table, const int* slot_mapping, int max_pages, int page_size,
                     const void* weight, int ndtype, float eps, float* out, int T, int H, int vocab, int S,
                     cudaStream_t stream) {
    if (T <= 0) return kOk;
    if (H < 1 || vocab < 1 || S < 1 || S > kMaxStreams) {
        set_last_error("streams_embed: rows of %d, %d table rows, %d streams (at most %d)", H, vocab, S, kMaxStreams);
        return kBadShape;
    }
    if (bigram && (buckets < 1 || mul_prev < 0 || mul_cur < 0 || !token_ids || !block_table || !slot_mapping ||
                   !positions || !req_of_token || max_pages < 1 || page_size < 1)) {
        set_last_error("streams_embed: a second table of %lld rows needs its hash and the paged token ids",
                       (long long)buckets);
        return kBadShape;
    }
    const BigramArgs bg = {bigram, (long long)buckets, (long long)mul_prev, (long long)mul_cur, token_ids, block_table,
                           slot_mapping, max_pages, page_size};
    const bool vec = H % 4 == 0 && aligned16(table, bigram, out);
    MI_DISPATCH_2(wdtype, WT, ndtype, NT, {
        if (vec) launch_dependent(streams_embed_kernel<WT, NT, 4>, dim3(T), dim3(256), 0, stream, ids, positions,
                                  req_of_token, (const WT*)table, scale, bg, (const NT*)weight, eps, out, H, vocab, S);
        else launch_dependent(streams_embed_kernel<WT, NT, 1>, dim3(T), dim3(256), 0, stream, ids, positions,
                              req_of_token, (const WT*)table, scale, bg, (const NT*)weight, eps, out, H, vocab, S);
    });
    return finish_launch("streams_embed");
}

// xs [*, S, H] float; y [*, H] float or null (nothing is pending: the streams are read as they are); mix [S, S] (from,
// to), w_out [S], w_in [S] float; out [n, H]
int mi_streams_read(float* xs, const float* y, const float* mix, const float* w_out, const float* w_in,
                    const int* rows, const void* weight, int wdtype, void* out, int odtype, int n, int S, int H,
                    float eps, cudaStream_t stream) {
    if (n <= 0) return kOk;
    if (S < 1 || S > kMaxStreams || H < 1 || !w_in || !weight || (y && (!mix || !w_out))) {
        set_last_error("streams_read: %d streams (at most %d) of rows of %d, or a missing operand", S, kMaxStreams, H);
        return kBadShape;
    }
    const int vpt = (H / 4 + 255) / 256;
    if (S <= 4 && H % 4 == 0 && vpt <= 4 && aligned16(xs, y, weight, out)) {
#define MI_SR(SS, VV)                                                                                             \
    MI_DISPATCH_2(odtype, AT, wdtype, WT,                                                                         \
        launch_dependent(streams_read_vec_kernel<AT, WT, SS, VV>, dim3(n), dim3(256), 0, stream, xs, y, mix, w_out, \
                         w_in, rows, (const WT*)weight, (AT*)out, H, eps))
#define MI_SRS(SS)                                                                                                \
    do { if (vpt <= 1) { MI_SR(SS, 1); } else if (vpt <= 2) { MI_SR(SS, 2); } else { MI_SR(SS, 4); } } while (0)
        if (S == 1) MI_SRS(1);
        else if (S == 2) MI_SRS(2);
        else if (S == 3) MI_SRS(3);
        else MI_SRS(4);
#undef MI_SRS
#undef MI_SR
        return finish_launch("streams_read");
    }
    const size_t smem = sizeof(float) * (size_t)H;
    if (smem > 200 * 1024) { set_last_error("streams_read: rows of %d do not fit shared memory", H); return kBadShape; }
    MI_DISPATCH_2(odtype, AT, wdtype, WT, {
        if (smem > 40 * 1024)
            cudaFuncSetAttribute(streams_read_any_kernel<AT, WT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        launch_dependent(streams_read_any_kernel<AT, WT>, dim3(n), dim3(256), smem, stream, xs, y, mix, w_out, w_in,
                         rows, (const WT*)weight, (AT*)out, S, H, eps);
    });
    return finish_launch("streams_read");
}

int mi_streams_sum(const float* xs, const float* y, const float* mix, const float* w_out, float* out, int T, int S,
                   int H, cudaStream_t stream) {
    if (T <= 0) return kOk;
    if (S < 1 || H < 1 || (y && (!mix || !w_out))) {
        set_last_error("streams_sum: %d streams of rows of %d, or a missing operand", S, H);
        return kBadShape;
    }
    launch_dependent(streams_sum_kernel, dim3(T), dim3(256), 0, stream, xs, y, mix, w_out, out, S, H);
    return finish_launch("streams_sum");
}

int mi_relu_glu(const void* gu, void* out, int adtype, int64_t T, int I, cudaStream_t stream) {
    const int64_t total = T * I;
    if (total <= 0) return kOk;
    if (adtype == kBF16 && I % 8 == 0 && aligned16(gu, out)) {
        int64_t vblocks = (total / 8 + 255) / 256;
        if (vblocks > 148 * 16) vblocks = 148 * 16;
        launch_dependent(relu_glu_bf16x8_kernel, dim3((unsigned)vblocks), dim3(256), 0, stream, (const uint4*)gu,
                         (uint4*)out, total / 8, I / 8);
        return finish_launch("relu_glu");
    }
    int64_t blocks = (total + 255) / 256;
    if (blocks > 148 * 32) blocks = 148 * 32;
    MI_DISPATCH_1(adtype, AT,
        launch_dependent(relu_glu_kernel<AT>, dim3((unsigned)blocks), dim3(256), 0, stream, (const AT*)gu, (AT*)out,
                         total, I));
    return finish_launch("relu_glu");
}

}  // extern "C"
