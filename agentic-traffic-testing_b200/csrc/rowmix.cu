// Row kernels in which a token reads its predecessor, and a feed-forward activation with row statistics:
//   * embedding rows plus a row of a second table chosen by a hash of (previous token, token),
//   * token shift: the normed row blended with the previous position's normed row, per channel,
//   * a polynomial of unit-rms powers of the feed-forward's hidden row,
//   * the residual update of a parallel layer: stream + scale * (dense sublayer output + weighted expert outputs), embedding row
//     and pass vector where a block of layers is entered, and the one or two norms of the next layer, in one pass over the row.
// The predecessor of a step's first row comes from the sequence's state slot (the last token id; the last normed row of
// every layer), which the CTA that read it then overwrites with the step's last row: reader and writer are the same
// threads, so no second launch is needed. A sequence at position 0 has no predecessor whatever its slot holds.
// A step is a flat batch of rows; sequence s owns rows [seq_start[s], seq_start[s] + seq_count[s]), first position
// seq_pos0[s], state slot seq_slot[s]; tok_seq[t] is the sequence of row t (-1: padded row, skipped).
#include "common.cuh"

#include "../../include/atx_b200.h"

namespace atx {

template <typename XT>
__device__ __forceinline__ float rld(const XT* p, long long i);
template <>
__device__ __forceinline__ float rld<float>(const float* p, long long i) {
    return p[i];
}
template <>
__device__ __forceinline__ float rld<__nv_bfloat16>(const __nv_bfloat16* p, long long i) {
    return __bfloat162float(p[i]);
}
__device__ __forceinline__ void rst(float* p, long long i, float v) { p[i] = v; }
__device__ __forceinline__ void rst(__nv_bfloat16* p, long long i, float v) { p[i] = __float2bfloat16_rn(v); }
__device__ __forceinline__ float4 rld4(const float* p, long long i4) { return reinterpret_cast<const float4*>(p)[i4]; }
__device__ __forceinline__ float4 rld4(const __nv_bfloat16* p, long long i4) {
    const uint2 u = reinterpret_cast<const uint2*>(p)[i4];
    return make_float4(bf16lo(u.x), bf16hi(u.x), bf16lo(u.y), bf16hi(u.y));
}
__device__ __forceinline__ void rst4(float* p, long long i4, float4 v) { reinterpret_cast<float4*>(p)[i4] = v; }
__device__ __forceinline__ void rst4(__nv_bfloat16* p, long long i4, float4 v) {
    reinterpret_cast<uint2*>(p)[i4] = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}

// Four elements as they are stored (bf16: two registers instead of four).
template <typename XT>
struct Raw4;
template <>
struct Raw4<float> {
    float4 r;
    __device__ __forceinline__ void load(const float* p, long long i4) { r = reinterpret_cast<const float4*>(p)[i4]; }
    __device__ __forceinline__ float4 get() const { return r; }
};
template <>
struct Raw4<__nv_bfloat16> {
    uint2 r;
    __device__ __forceinline__ void load(const __nv_bfloat16* p, long long i4) { r = reinterpret_cast<const uint2*>(p)[i4]; }
    __device__ __forceinline__ float4 get() const { return make_float4(bf16lo(r.x), bf16hi(r.x), bf16lo(r.y), bf16hi(r.y)); }
};

static void set_pdl_row(cudaLaunchConfig_t& cfg, cudaLaunchAttribute* attr, int flags) {
    if (flags & ATX_FLAG_PDL) {
        attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[0].val.programmaticStreamSerializationAllowed = 1;
        cfg.attrs = attr;
        cfg.numAttrs = 1;
    }
}

#define ATX_ROW_XT(dtype_, ...)                \
    do {                                       \
        if ((dtype_) == ATX_DT_F32) {          \
            using XT = float;                  \
            __VA_ARGS__;                       \
        } else {                               \
            using XT = __nv_bfloat16;          \
            __VA_ARGS__;                       \
        }                                      \
    } while (0)

// ---- embedding row + pair-table row -----------------------------------------------------------------------------------
// out[t] = table[id_t] * scale + pair[(id_(t-1) * mul_prev + id_t * mul_cur) mod buckets]; a sequence's first token takes
// row `buckets` (the table has buckets + 1 rows). prev_tok [slots]: the last token of every live sequence.
template <typename XT>
__global__ void __launch_bounds__(128)
embed_rows_pair_kernel(const int* __restrict__ ids, const XT* __restrict__ table, float scale, const XT* __restrict__ pair,
                       int buckets, int mul_prev, int mul_cur, int* __restrict__ prev_tok, const int* __restrict__ tok_seq,
                       const int* __restrict__ seq_start, const int* __restrict__ seq_count,
                       const int* __restrict__ seq_pos0, const int* __restrict__ seq_slot, float* __restrict__ out, int W,
                       int V) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int s = tok_seq[t];
    float* dst = out + static_cast<long long>(t) * W;
    if (s < 0) {   // padded row: defined contents, no state
        for (int i = threadIdx.x; i < W; i += blockDim.x) dst[i] = 0.f;
        return;
    }
    auto clamp = [V](int id) { return id < 0 ? 0 : (id >= V ? V - 1 : id); };
    const int id = clamp(ids[t]);
    const int r0 = seq_start[s];
    long long prow = buckets;
    if (t != r0) {
        prow = (static_cast<long long>(clamp(ids[t - 1])) * mul_prev + static_cast<long long>(id) * mul_cur) % buckets;
    } else {
        const int slot = seq_slot[s];
        if (seq_pos0[s] > 0)
            prow = (static_cast<long long>(clamp(prev_tok[slot])) * mul_prev + static_cast<long long>(id) * mul_cur) % buckets;
        __syncthreads();   // every thread has read the slot
        if (threadIdx.x == 0) prev_tok[slot] = ids[r0 + seq_count[s] - 1];
    }
    const XT* src = table + static_cast<long long>(id) * W;
    const XT* ps = pair + prow * W;
    if ((W & 3) == 0 && ((reinterpret_cast<unsigned long long>(table) | reinterpret_cast<unsigned long long>(pair) |
                          reinterpret_cast<unsigned long long>(out)) & 15) == 0) {
#pragma unroll 4
        for (int i = threadIdx.x; i < W / 4; i += blockDim.x) {
            const float4 a = rld4(src, i), b = rld4(ps, i);
            rst4(dst, i, make_float4(fmaf(a.x, scale, b.x), fmaf(a.y, scale, b.y), fmaf(a.z, scale, b.z), fmaf(a.w, scale, b.w)));
        }
        return;
    }
    for (int i = threadIdx.x; i < W; i += blockDim.x) dst[i] = fmaf(rld(src, i), scale, rld(ps, i));
}

// ---- token shift ----------------------------------------------------------------------------------------------------------
// out[t] = x[t] + (x[t-1] - x[t]) * mu, x fp32 (the normed rows), out of the element type; state [slots, W] fp32 keeps
// the last x of every live sequence.
template <typename XT>
__global__ void __launch_bounds__(256)
token_shift_kernel(const float* __restrict__ x, const XT* __restrict__ mu, float* __restrict__ state,
                   const int* __restrict__ tok_seq, const int* __restrict__ seq_start, const int* __restrict__ seq_count,
                   const int* __restrict__ seq_pos0, const int* __restrict__ seq_slot, XT* __restrict__ out, int W) {
    pdl_launch_dependents();
    pdl_wait();
    const long long t = blockIdx.x;
    const int s = tok_seq[t];
    XT* o = out + t * W;
    if (s < 0) {
        for (int i = threadIdx.x; i < W; i += blockDim.x) rst(o, i, 0.f);
        return;
    }
    const int r0 = seq_start[s];
    const bool first = t == r0;
    const bool none = first && seq_pos0[s] == 0;
    const float* cur = x + t * W;
    const float* prev = first ? state + static_cast<long long>(seq_slot[s]) * W : cur - W;
    float* keep = first ? state + static_cast<long long>(seq_slot[s]) * W : nullptr;
    const float* last = x + (static_cast<long long>(r0) + seq_count[s] - 1) * W;   // the step's last row of the sequence
    if ((W & 3) == 0 && ((reinterpret_cast<unsigned long long>(x) | reinterpret_cast<unsigned long long>(mu) |
                          reinterpret_cast<unsigned long long>(state) | reinterpret_cast<unsigned long long>(out)) & 15) == 0) {
#pragma unroll 2
        for (int i = threadIdx.x; i < W / 4; i += blockDim.x) {
            const float4 c = rld4(cur, i), m = rld4(mu, i);
            const float4 p = none ? make_float4(0.f, 0.f, 0.f, 0.f) : rld4(prev, i);
            rst4(o, i, make_float4(fmaf(p.x - c.x, m.x, c.x), fmaf(p.y - c.y, m.y, c.y), fmaf(p.z - c.z, m.z, c.z),
                                   fmaf(p.w - c.w, m.w, c.w)));
            if (keep) rst4(keep, i, rld4(last, i));   // the same thread read this part of the slot above
        }
        return;
    }
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
        const float c = cur[i], p = none ? 0.f : prev[i];
        rst(o, i, fmaf(p - c, rld(mu, i), c));
        if (keep) keep[i] = last[i];
    }
}

// ---- polynomial of unit-rms powers -------------------------------------------------------------------------------------------
// out = a z / rms(z) + b z^2 / rms(z^2) + c z^3 / rms(z^3) + e over a row of F elements; coef = {a, b, c, e} fp32.
template <typename XT>
__global__ void __launch_bounds__(256)
poly_norm_act_kernel(const float* __restrict__ z, long long ldz, const float* __restrict__ coef, XT* __restrict__ out,
                     long long ldo, int F, float eps) {
    __shared__ float red[3][8];
    pdl_launch_dependents();
    const float a = coef[0], b = coef[1], c = coef[2], e = coef[3];
    pdl_wait();
    const long long t = blockIdx.x;
    const float* zr = z + t * ldz;
    XT* o = out + t * ldo;
    const bool vec = (F & 3) == 0 && (ldz & 3) == 0 && (ldo & 3) == 0 &&
                     ((reinterpret_cast<unsigned long long>(z) | reinterpret_cast<unsigned long long>(out)) & 15) == 0;
    float s2 = 0.f, s4 = 0.f, s6 = 0.f;
    auto take = [&](float v) {
        const float v2 = v * v;
        s2 += v2;
        s4 = fmaf(v2, v2, s4);
        s6 = fmaf(v2 * v2, v2, s6);
    };
    if (vec) {
        for (int i = threadIdx.x; i < F / 4; i += blockDim.x) {
            const float4 v = rld4(zr, i);
            take(v.x), take(v.y), take(v.z), take(v.w);
        }
    } else {
        for (int i = threadIdx.x; i < F; i += blockDim.x) take(zr[i]);
    }
    s2 = warp_sum(s2), s4 = warp_sum(s4), s6 = warp_sum(s6);
    if ((threadIdx.x & 31) == 0) {
        red[0][threadIdx.x >> 5] = s2;
        red[1][threadIdx.x >> 5] = s4;
        red[2][threadIdx.x >> 5] = s6;
    }
    __syncthreads();
    s2 = s4 = s6 = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) s2 += red[0][i], s4 += red[1][i], s6 += red[2][i];
    const float inv = 1.f / static_cast<float>(F);
    const float r1 = a * rsqrtf(s2 * inv + eps), r2 = b * rsqrtf(s4 * inv + eps), r3 = c * rsqrtf(s6 * inv + eps);
    auto act = [&](float v) { return fmaf(v, fmaf(v, fmaf(v, r3, r2), r1), e); };   // ((r3 v + r2) v + r1) v + e
    if (vec) {
        for (int i = threadIdx.x; i < F / 4; i += blockDim.x) {
            const float4 v = rld4(zr, i);
            rst4(o, i, make_float4(act(v.x), act(v.y), act(v.z), act(v.w)));
        }
    } else {
        for (int i = threadIdx.x; i < F; i += blockDim.x) rst(o, i, act(zr[i]));
    }
}

// ---- residual update of a parallel layer ------------------------------------------------------------------------------------
// Per row t (r = rows ? rows[t] : t):
//   v = h[r] (or the embedding row, table_mode 2; its RMS norm times table_w, if given) + y_scale * (y[r] + sum_k wgt[r, k] experts[slot_of[r, k]])
//       + embedding row (table_mode 1) + vec;         h[r] = v (not with rows)
//   out_x[t] = v / sqrt(mean(v^2) + eps) * (w_shift + w_x)     x = a, b
// Both norms share the row's statistic. CTAs beyond T clear zero_ptr. NV > 0: NV vectors of four elements per thread, the row
// stays in registers; NV = 0: any width and alignment, the row staged in shared memory.
struct ParallelResidArgs {
    float* h;
    atx_resid_terms tm;
    const void* w_a;
    void* out_a;
    const void* w_b;
    void* out_b;
    float w_shift, eps;
    const int* rows;
    int T, W;
    uint4* zero_ptr;
    long long zero_vecs;
};
constexpr int kResidTopMax = 64;

__device__ __forceinline__ float row_sum(float v, float* red) {   // over the CTA; every thread gets the result
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
    const int nw = (blockDim.x + 31) >> 5;
    for (int i = 0; i < nw; ++i) t += red[i];
    return t;
}

template <typename XT, int NV>
__global__ void __launch_bounds__(NV == 8 ? 512 : 1024)
parallel_resid_norm_kernel(const __grid_constant__ ParallelResidArgs a) {
    extern __shared__ __align__(16) float srow_p[];
    __shared__ float red[32];
    __shared__ float s_w[kResidTopMax];
    __shared__ long long s_row[kResidTopMax];
    pdl_launch_dependents();
    const int W = a.W, W4 = W / 4;
    const XT* wa = reinterpret_cast<const XT*>(a.w_a);
    const XT* wb = reinterpret_cast<const XT*>(a.w_b);
    const XT* vec = reinterpret_cast<const XT*>(a.tm.vec);
    // one vector per thread (decode-sized steps): the weights, which no kernel writes, are fetched ahead of the wait
    float4 wa4 = make_float4(0.f, 0.f, 0.f, 0.f), wb4 = wa4, vc4 = wa4;
    if (NV == 1 && static_cast<int>(threadIdx.x) < W4 && static_cast<int>(blockIdx.x) < a.T) {
        if (wa) wa4 = rld4(wa, threadIdx.x);
        if (wb) wb4 = rld4(wb, threadIdx.x);
        if (vec) vc4 = rld4(vec, threadIdx.x);
    }
    pdl_wait();
    if (static_cast<int>(blockIdx.x) >= a.T) {
        const long long nb = gridDim.x - a.T;
        for (long long i = static_cast<long long>(blockIdx.x - a.T) * blockDim.x + threadIdx.x; i < a.zero_vecs;
             i += nb * blockDim.x)
            a.zero_ptr[i] = make_uint4(0, 0, 0, 0);
        return;
    }
    const int t = blockIdx.x;
    const long long r = a.rows ? a.rows[t] : t;
    float* hr = a.h + r * W;
    float* yr = a.tm.y ? a.tm.y + r * W : nullptr;
    const int top = a.tm.experts ? a.tm.top : 0;
    if (top) {
        for (int k = threadIdx.x; k < top; k += blockDim.x) {
            const int slot = a.tm.slot_of[r * top + k];
            s_w[k] = slot >= 0 ? a.tm.wgt[r * top + k] : 0.f;
            s_row[k] = slot >= 0 ? static_cast<long long>(slot) * a.tm.lde : -1;
        }
        __syncthreads();
    }
    const XT* er = nullptr;
    if (a.tm.table_mode) {
        int id = a.tm.ids[r];
        id = id < 0 ? 0 : (id >= a.tm.vocab ? a.tm.vocab - 1 : id);
        er = reinterpret_cast<const XT*>(a.tm.table) + static_cast<long long>(id) * W;
    }
    const bool start = a.tm.table_mode == 2, enter = a.tm.table_mode == 1;
    const XT* tw = start ? reinterpret_cast<const XT*>(a.tm.table_w) : nullptr;
    float rs0 = 1.f;   // of the embedding row that the stream starts as
    const bool store = !a.rows && (yr || top || er || vec);
    const float sc = a.tm.y_scale;
    float ss = 0.f;
    if constexpr (NV > 0) {
        // Every loop below issues its NV loads before anything uses or stores one of them.
        float4 v[NV];
        Raw4<XT> ga[NV], gb[NV];
        bool on[NV];
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = threadIdx.x + n * blockDim.x;
            on[n] = i < W4;
            v[n] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (on[n]) v[n] = start ? rld4(er, i) : rld4(hr, i);
        }
        if (NV > 1) {   // the norm weights are on their way while the row is summed
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                const int i = threadIdx.x + n * blockDim.x;
                if (wa && on[n]) ga[n].load(wa, i);
                if (wb && on[n]) gb[n].load(wb, i);
            }
        }
        if (tw) {
            float s0 = 0.f;
#pragma unroll
            for (int n = 0; n < NV; ++n) s0 += v[n].x * v[n].x + v[n].y * v[n].y + v[n].z * v[n].z + v[n].w * v[n].w;
            rs0 = rsqrtf(row_sum(s0, red) / static_cast<float>(W) + a.eps);
            __syncthreads();   // red is used again for the outgoing norm
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                if (!on[n]) continue;
                const float4 g = rld4(tw, threadIdx.x + n * blockDim.x);
                v[n].x *= rs0 * g.x, v[n].y *= rs0 * g.y, v[n].z *= rs0 * g.z, v[n].w *= rs0 * g.w;
            }
        }
        auto add_row = [&](const float* src, float w) {
            float4 e[NV];
#pragma unroll
            for (int n = 0; n < NV; ++n)
                e[n] = on[n] ? rld4(src, threadIdx.x + n * blockDim.x) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                v[n].x = fmaf(w, e[n].x, v[n].x), v[n].y = fmaf(w, e[n].y, v[n].y);
                v[n].z = fmaf(w, e[n].z, v[n].z), v[n].w = fmaf(w, e[n].w, v[n].w);
            }
        };
        if (yr) {
            add_row(yr, sc);
            if (a.tm.zero_y) {
#pragma unroll
                for (int n = 0; n < NV; ++n)
                    if (on[n]) rst4(yr, threadIdx.x + n * blockDim.x, make_float4(0.f, 0.f, 0.f, 0.f));
            }
        }
        for (int k = 0; k < top; ++k)
            if (s_row[k] >= 0) add_row(a.tm.experts + s_row[k], sc * s_w[k]);
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = threadIdx.x + n * blockDim.x;
            if (!on[n]) continue;
            if (enter) {
                const float4 e = rld4(er, i);
                v[n].x += e.x, v[n].y += e.y, v[n].z += e.z, v[n].w += e.w;
            }
            if (vec) {
                const float4 c = NV == 1 ? vc4 : rld4(vec, i);
                v[n].x += c.x, v[n].y += c.y, v[n].z += c.z, v[n].w += c.w;
            }
            if (store) rst4(hr, i, v[n]);
            ss += v[n].x * v[n].x + v[n].y * v[n].y + v[n].z * v[n].z + v[n].w * v[n].w;
        }
        if (!a.out_a && !a.out_b) return;
        const float rs = rsqrtf(row_sum(ss, red) / static_cast<float>(W) + a.eps), sh = a.w_shift;
        XT* oa = reinterpret_cast<XT*>(a.out_a) + static_cast<long long>(t) * W;
        XT* ob = reinterpret_cast<XT*>(a.out_b) + static_cast<long long>(t) * W;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int i = threadIdx.x + n * blockDim.x;
            if (!on[n]) continue;
            const float4 u = make_float4(v[n].x * rs, v[n].y * rs, v[n].z * rs, v[n].w * rs);
            if (a.out_a) {
                const float4 g = NV == 1 ? wa4 : ga[n].get();
                rst4(oa, i, make_float4(u.x * (sh + g.x), u.y * (sh + g.y), u.z * (sh + g.z), u.w * (sh + g.w)));
            }
            if (a.out_b) {
                const float4 g = NV == 1 ? wb4 : gb[n].get();
                rst4(ob, i, make_float4(u.x * (sh + g.x), u.y * (sh + g.y), u.z * (sh + g.z), u.w * (sh + g.w)));
            }
        }
    } else {
        if (tw) {
            float s0 = 0.f;
            for (int i = threadIdx.x; i < W; i += blockDim.x) {
                const float e = rld(er, i);
                s0 += e * e;
            }
            rs0 = rsqrtf(row_sum(s0, red) / static_cast<float>(W) + a.eps);
            __syncthreads();
        }
        for (int i = threadIdx.x; i < W; i += blockDim.x) {
            float v = start ? rld(er, i) : hr[i], add = 0.f;
            if (tw) v *= rs0 * rld(tw, i);
            if (yr) {
                add = yr[i];
                if (a.tm.zero_y) yr[i] = 0.f;
            }
            for (int k = 0; k < top; ++k)
                if (s_row[k] >= 0) add = fmaf(s_w[k], a.tm.experts[s_row[k] + i], add);
            v = fmaf(sc, add, v);
            if (enter) v += rld(er, i);
            if (vec) v += rld(vec, i);
            if (store) hr[i] = v;
            srow_p[i] = v;
            ss += v * v;
        }
        if (!a.out_a && !a.out_b) return;
        const float rs = rsqrtf(row_sum(ss, red) / static_cast<float>(W) + a.eps);
        XT* oa = reinterpret_cast<XT*>(a.out_a) + static_cast<long long>(t) * W;
        XT* ob = reinterpret_cast<XT*>(a.out_b) + static_cast<long long>(t) * W;
        for (int i = threadIdx.x; i < W; i += blockDim.x) {   // each thread re-reads what it wrote itself
            const float u = srow_p[i] * rs;
            if (a.out_a) rst(oa, i, u * (a.w_shift + rld(wa, i)));
            if (a.out_b) rst(ob, i, u * (a.w_shift + rld(wb, i)));
        }
    }
}

}  // namespace atx

using namespace atx;

extern "C" {

int atx_embed_rows_pair(const int* ids, const void* table, float scale, const void* pair_table, int buckets, int mul_prev,
                        int mul_cur, int* prev_tok, const int* tok_seq, const int* seq_start, const int* seq_count,
                        const int* seq_pos0, const int* seq_slot, float* out, int T, int W, int V, int dtype, int flags,
                        atx_stream_t stream) {
    ATX_REQUIRE(ids && table && pair_table && prev_tok && tok_seq && seq_start && seq_count && seq_pos0 && seq_slot && out,
                "atx_embed_rows_pair: null pointer");
    ATX_REQUIRE(T > 0 && W > 0 && V > 0 && buckets > 0, "atx_embed_rows_pair: bad shape T=%d W=%d V=%d buckets=%d", T, W, V,
                buckets);
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    cfg.gridDim = dim3(T);
    cfg.blockDim = dim3(128);
    cfg.stream = reinterpret_cast<cudaStream_t>(stream);
    set_pdl_row(cfg, attr, flags);
    ATX_ROW_XT(dtype, ATX_CUDA(cudaLaunchKernelEx(&cfg, embed_rows_pair_kernel<XT>, ids, reinterpret_cast<const XT*>(table),
                                                  scale, reinterpret_cast<const XT*>(pair_table), buckets, mul_prev, mul_cur,
                                                  prev_tok, tok_seq, seq_start, seq_count, seq_pos0, seq_slot, out, W, V)));
    return ATX_OK;
}

int atx_token_shift(const float* x, const void* mu, float* state, const int* tok_seq, const int* seq_start,
                    const int* seq_count, const int* seq_pos0, const int* seq_slot, void* out, int T, int W, int dtype,
                    int flags, atx_stream_t stream) {
    ATX_REQUIRE(x && mu && state && tok_seq && seq_start && seq_count && seq_pos0 && seq_slot && out,
                "atx_token_shift: null pointer");
    ATX_REQUIRE(T > 0 && W > 0, "atx_token_shift: bad shape T=%d W=%d", T, W);
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    cfg.gridDim = dim3(T);
    cfg.blockDim = dim3(256);
    cfg.stream = reinterpret_cast<cudaStream_t>(stream);
    set_pdl_row(cfg, attr, flags);
    ATX_ROW_XT(dtype, ATX_CUDA(cudaLaunchKernelEx(&cfg, token_shift_kernel<XT>, x, reinterpret_cast<const XT*>(mu), state,
                                                  tok_seq, seq_start, seq_count, seq_pos0, seq_slot,
                                                  reinterpret_cast<XT*>(out), W)));
    return ATX_OK;
}

int atx_poly_norm_act(const float* z, long long ldz, const float* coef, void* out, long long ldo, int T, int F, float eps,
                      int dtype, int flags, atx_stream_t stream) {
    ATX_REQUIRE(z && coef && out, "atx_poly_norm_act: null pointer");
    ATX_REQUIRE(T > 0 && F > 0 && ldz >= F && ldo >= F, "atx_poly_norm_act: bad shape T=%d F=%d ldz=%lld ldo=%lld", T, F, ldz,
                ldo);
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    cfg.gridDim = dim3(T);
    cfg.blockDim = dim3(256);
    cfg.stream = reinterpret_cast<cudaStream_t>(stream);
    set_pdl_row(cfg, attr, flags);
    ATX_ROW_XT(dtype, ATX_CUDA(cudaLaunchKernelEx(&cfg, poly_norm_act_kernel<XT>, z, ldz, coef, reinterpret_cast<XT*>(out), ldo,
                                                  F, eps)));
    return ATX_OK;
}

int atx_parallel_resid_norm(float* h, const atx_resid_terms* terms, const void* w_a, void* out_a, const void* w_b, void* out_b,
                            float w_shift, const int* rows, int T, int W, float eps, void* zero_ptr, long long zero_bytes,
                            int dtype, int flags, atx_stream_t stream) {
    ATX_REQUIRE(h && terms, "atx_parallel_resid_norm: null pointer");
    const atx_resid_terms& tm = *terms;
    ATX_REQUIRE(T > 0 && W > 0 && W <= 12288, "atx_parallel_resid_norm: bad shape T=%d W=%d (W <= 12288)", T, W);
    ATX_REQUIRE((w_a == nullptr) == (out_a == nullptr) && (w_b == nullptr) == (out_b == nullptr),
                "atx_parallel_resid_norm: a norm weight and its output come together");
    ATX_REQUIRE(!tm.experts || (tm.wgt && tm.slot_of && tm.top > 0 && tm.top <= kResidTopMax && tm.lde >= W),
                "atx_parallel_resid_norm: experts need weights, slots and 1..%d choices (got %d)", kResidTopMax, tm.top);
    ATX_REQUIRE(tm.table_mode >= 0 && tm.table_mode <= 2 && (tm.table_mode == 0 || (tm.ids && tm.table && tm.vocab > 0)),
                "atx_parallel_resid_norm: table_mode=%d needs ids and a table", tm.table_mode);
    ATX_REQUIRE(zero_bytes >= 0 && zero_bytes % 16 == 0 && (zero_bytes == 0 || zero_ptr) && !(tm.zero_y && rows),
                "atx_parallel_resid_norm: zero_bytes=%lld must be a non-negative multiple of 16 with a buffer; zero_y not with rows",
                zero_bytes);
    ParallelResidArgs a = {h, tm, w_a, out_a, w_b, out_b, w_shift, eps, rows, T, W, reinterpret_cast<uint4*>(zero_ptr), zero_bytes / 16};
    auto al16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const bool v4 = W % 4 == 0 && al16(h) && al16(tm.y) && al16(tm.experts) && (!tm.experts || tm.lde % 4 == 0) && al16(tm.table) &&
                    al16(tm.table_w) && al16(tm.vec) && al16(w_a) && al16(out_a) && al16(w_b) && al16(out_b);
    // few rows: as many threads per row as it has vectors; many rows: 256 threads and several vectors each
    const int W4 = W / 4;
    const int want = T <= 512 ? (W4 + 31) / 32 * 32 : 256;
    int threads = want > 1024 ? 1024 : (want < 64 ? 64 : want);
    while ((W4 + threads - 1) / threads > 8) threads *= 2;
    const int nv = (W4 + threads - 1) / threads;
    long long zb = (a.zero_vecs + 256 * 8 - 1) / (256 * 8);
    if (zb > 2048) zb = 2048;
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    cfg.gridDim = dim3(static_cast<unsigned>(T + zb));
    cfg.blockDim = dim3(v4 ? threads : 256);
    cfg.dynamicSmemBytes = v4 ? 0 : static_cast<size_t>(W) * 4;
    cfg.stream = reinterpret_cast<cudaStream_t>(stream);
    set_pdl_row(cfg, attr, flags);
#define ATX_PAR_RESID(NV_) ATX_ROW_XT(dtype, ATX_CUDA(cudaLaunchKernelEx(&cfg, parallel_resid_norm_kernel<XT, NV_>, a)))
    if (!v4)
        ATX_PAR_RESID(0);
    else if (nv <= 1)
        ATX_PAR_RESID(1);
    else if (nv == 2)
        ATX_PAR_RESID(2);
    else if (nv <= 4)
        ATX_PAR_RESID(4);
    else
        ATX_PAR_RESID(8);
#undef ATX_PAR_RESID
    return ATX_OK;
}

}  // extern "C"
