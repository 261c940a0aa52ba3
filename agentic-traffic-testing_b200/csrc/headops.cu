// Per-head and element-wise operations that sit between a model's projections and its attention kernels:
//   * the element-wise squashing norm  out = tanh(alpha x) w + b  (no row statistics; optional row gather),
//   * a unary activation between the two feed-forward GEMMs (squared ReLU, tanh-GELU),
//   * "head preparation": slices of a fused projection row are cut into heads, each head optionally RMS-normed over its
//     leading elements, rotated in adjacent pairs over a sub-range, blended with the same token's values of an earlier
//     layer, and written either to a row buffer (queries, GEMM inputs) or into the paged cache at the token's slot.
//     A launch takes up to four such slices, so that q, k and v of a layer (or the two bottlenecks of a latent
//     attention) are prepared together,
//   * the same for slices that first pass a short causal convolution over time, per channel, whose carried inputs live in
//     the sequence's state slot; the convolved head can be kept as it is (values that are the keys) beside the rotated and
//     normed one,
//   * a cap on logits, c tanh(z / c), in place,
//   * a small matrix product per head  out[t, h, :] = W_h x[t, h, :]  with an optional sigmoid gate per output element
//     (the per-head up-projections of latent attention in its absorbed form).
// Element type XT (weights, GEMM inputs, pages) = bf16 or fp32; sums, norms, rotations and blends are fp32.
#include "common.cuh"

#include "../../include/atx_b200.h"

namespace atx {

template <typename XT>
__device__ __forceinline__ float hld(const XT* p, long long i);
template <>
__device__ __forceinline__ float hld<float>(const float* p, long long i) {
    return p[i];
}
template <>
__device__ __forceinline__ float hld<__nv_bfloat16>(const __nv_bfloat16* p, long long i) {
    return __bfloat162float(p[i]);
}
__device__ __forceinline__ void hst(float* p, long long i, float v) { p[i] = v; }
__device__ __forceinline__ void hst(__nv_bfloat16* p, long long i, float v) { p[i] = __float2bfloat16_rn(v); }

__device__ __forceinline__ float4 hld4(const float* p, long long i4) { return reinterpret_cast<const float4*>(p)[i4]; }
__device__ __forceinline__ float4 hld4(const __nv_bfloat16* p, long long i4) {
    const uint2 u = reinterpret_cast<const uint2*>(p)[i4];
    return make_float4(bf16lo(u.x), bf16hi(u.x), bf16lo(u.y), bf16hi(u.y));
}
__device__ __forceinline__ void hst4(float* p, long long i4, float4 v) { reinterpret_cast<float4*>(p)[i4] = v; }
__device__ __forceinline__ void hst4(__nv_bfloat16* p, long long i4, float4 v) {
    reinterpret_cast<uint2*>(p)[i4] = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}

static void set_pdl_attr(cudaLaunchConfig_t& cfg, cudaLaunchAttribute* attr, int flags) {
    if (flags & ATX_FLAG_PDL) {
        attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[0].val.programmaticStreamSerializationAllowed = 1;
        cfg.attrs = attr;
        cfg.numAttrs = 1;
    }
}

#define ATX_HEADOPS_XT(dtype, ...)       \
    do {                                 \
        if ((dtype) == ATX_DT_F32) {     \
            using XT = float;            \
            __VA_ARGS__;                 \
        } else {                         \
            using XT = __nv_bfloat16;    \
            __VA_ARGS__;                 \
        }                                \
    } while (0)

// ---- tanh norm ---------------------------------------------------------------------------------------------------------
// Blocks [0, T) take one row each; the blocks after them clear zero_ptr (the accumulator of a split-K GEMM that follows).
template <typename XT>
__global__ void __launch_bounds__(256)
tanh_norm_kernel(const float* __restrict__ x, const int* __restrict__ rows, float alpha, const XT* __restrict__ w,
                 const XT* __restrict__ b, XT* __restrict__ out, int T, int W, uint4* __restrict__ zero_ptr,
                 long long zero_vecs) {
    pdl_launch_dependents();
    if (static_cast<int>(blockIdx.x) >= T) {
        pdl_wait();   // a kernel of the previous layer may still be reading the buffer
        const long long nb = gridDim.x - T, b0 = blockIdx.x - T;
        for (long long i = b0 * blockDim.x + threadIdx.x; i < zero_vecs; i += nb * blockDim.x)
            zero_ptr[i] = make_uint4(0, 0, 0, 0);
        return;
    }
    pdl_wait();
    const int t = blockIdx.x;
    const long long r = rows ? rows[t] : t;
    const float* src = x + r * W;
    XT* dst = out + static_cast<long long>(t) * W;
    const bool vec = (W & 3) == 0 && ((reinterpret_cast<unsigned long long>(x) | reinterpret_cast<unsigned long long>(out) |
                                       reinterpret_cast<unsigned long long>(w) | reinterpret_cast<unsigned long long>(b)) & 15) == 0;
    if (vec) {
        for (int i = threadIdx.x; i < W / 4; i += blockDim.x) {
            const float4 v = hld4(src, i), g = hld4(w, i), c = hld4(b, i);
            float4 o;
            o.x = fmaf(tanhf(alpha * v.x), g.x, c.x);
            o.y = fmaf(tanhf(alpha * v.y), g.y, c.y);
            o.z = fmaf(tanhf(alpha * v.z), g.z, c.z);
            o.w = fmaf(tanhf(alpha * v.w), g.w, c.w);
            hst4(dst, i, o);
        }
        return;
    }
    for (int i = threadIdx.x; i < W; i += blockDim.x) hst(dst, i, fmaf(tanhf(alpha * src[i]), hld(w, i), hld(b, i)));
}

// ---- unary activation ---------------------------------------------------------------------------------------------------
__device__ __forceinline__ float unary_act(float z, int kind) {
    if (kind == ATX_ACT_RELU2) {
        const float r = fmaxf(z, 0.f);
        return r * r;
    }
    // tanh form of GELU: z/2 (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return 0.5f * z * (1.f + tanhf(u));
}

template <typename XT>
__global__ void __launch_bounds__(256)
unary_act_kernel(const float* __restrict__ in, long long ldi, XT* __restrict__ out, long long ldo, int T, int I, int kind) {
    pdl_launch_dependents();
    pdl_wait();
    const long long n = static_cast<long long>(T) * I;
    for (long long e = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; e < n;
         e += static_cast<long long>(gridDim.x) * blockDim.x) {
        const long long t = e / I;
        const int i = static_cast<int>(e - t * I);
        hst(out, t * ldo + i, unary_act(in[t * ldi + i], kind));
    }
}

// ---- head preparation ----------------------------------------------------------------------------------------------------
struct PrepArgs {
    int n;
    int total_heads;
    atx_head_seg seg[ATX_HEAD_SEGS_MAX];
};

// One warp per (row, head); WIDE: one CTA per (row, head), for steps of few rows whose heads are wide (a bottleneck of
// a thousand elements normed by one warp is a chain of dependent loads). A lane owns single elements (or four); a rotated
// element also reads its partner of the pair.
template <typename XT, bool WIDE>
__global__ void __launch_bounds__(256)
head_prepare_kernel(const float* __restrict__ src, long long ld, const int* __restrict__ positions,
                    const int* __restrict__ slots, int T, int bs, float eps, const __grid_constant__ PrepArgs a) {
    __shared__ float red[8];
    pdl_launch_dependents();
    pdl_wait();
    constexpr int kStep = WIDE ? 256 : 32;
    const int lane = WIDE ? threadIdx.x : (threadIdx.x & 31);
    const long long wid = WIDE ? static_cast<long long>(blockIdx.x)
                               : static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
    auto head_sum = [&](float v) -> float {   // over the threads that share the head
        v = warp_sum(v);
        if constexpr (WIDE) {
            if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
            __syncthreads();
            v = 0.f;
#pragma unroll
            for (int i = 0; i < 8; ++i) v += red[i];
        }
        return v;
    };
    if (wid >= static_cast<long long>(T) * a.total_heads) return;
    const long long t = wid / a.total_heads;
    int hh = static_cast<int>(wid - t * a.total_heads);
    int si = 0;
    while (si + 1 < a.n && hh >= a.seg[si].heads) {
        hh -= a.seg[si].heads;
        ++si;
    }
    const atx_head_seg& s = a.seg[si];
    const int slot = slots ? slots[t] : 0;
    if (slot < 0) return;   // padded row
    const float* x = src + t * ld + s.src_off + static_cast<long long>(hh) * s.src_stride;
    const XT* nw = reinterpret_cast<const XT*>(s.norm_w);
    float r = 1.f;
    const float* cs = nullptr;
    const int half = s.rot_dims / 2;
    if (s.rot_dims > 0) cs = s.rot + static_cast<long long>(positions[t]) * s.rot_dims;
    XT* dst;
    if (s.dst_kind == ATX_HEAD_DST_PAGES) {
        const int blk = slot / bs, off = slot - blk * bs;
        dst = reinterpret_cast<XT*>(s.dst) +
              ((static_cast<long long>(blk) * s.heads + hh) * bs + off) * s.dst_stride + s.dst_off;
    } else {
        dst = reinterpret_cast<XT*>(s.dst) + t * s.dst_ld + s.dst_off + static_cast<long long>(hh) * s.dst_stride;
    }
    const long long flat = (t * s.heads + hh) * s.width;   // index into mix_src / save
    // Four elements per access where every offset, pitch and count of the slice is a multiple of four and the pointers
    // are aligned: a rotated pair then lies inside one access, so no partner has to be fetched.
    const bool vec =
        ((s.width | s.src_off | s.src_stride | s.norm_dims | s.rot_off | s.dst_off | s.dst_stride) & 3) == 0 && (ld & 3) == 0 &&
        (s.dst_kind == ATX_HEAD_DST_PAGES || (s.dst_ld & 3) == 0) &&
        ((reinterpret_cast<unsigned long long>(src) | reinterpret_cast<unsigned long long>(s.dst) |
          reinterpret_cast<unsigned long long>(s.norm_w) | reinterpret_cast<unsigned long long>(s.mix_src) |
          reinterpret_cast<unsigned long long>(s.save)) & 15) == 0 &&
        (!s.rot_half || (half & 3) == 0);   // half-split pairs: the partner's four elements are one more aligned access
    if (vec) {
        if (s.norm_dims > 0) {
            float ss = 0.f;
#pragma unroll 4
            for (int i4 = lane; i4 < s.norm_dims / 4; i4 += kStep) {
                const float4 v = hld4(x, i4);
                ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
            }
            ss = head_sum(ss);
            r = rsqrtf(ss / static_cast<float>(s.norm_dims) + eps);
        }
#pragma unroll 2
        for (int i4 = lane; i4 < s.width / 4; i4 += kStep) {
            const float4 v = hld4(x, i4);
            float e[4] = {v.x, v.y, v.z, v.w};
            const int i = 4 * i4;
            if (i < s.norm_dims) {
                const float4 g = hld4(nw, i4);
                e[0] *= r * g.x, e[1] *= r * g.y, e[2] *= r * g.z, e[3] *= r * g.w;
            }
            if (s.rot_half) {
                // element j < half pairs with j + half: (u, w) -> (u c - w s, w c + u s), angle index j mod half
                const int j = i - s.rot_off;
                if (j >= 0 && j < s.rot_dims) {
                    const bool low = j < half;
                    const int ip4 = low ? i4 + half / 4 : i4 - half / 4;
                    const float4 pv = hld4(x, ip4);
                    float pe[4] = {pv.x, pv.y, pv.z, pv.w};
                    if (4 * ip4 < s.norm_dims) {
                        const float4 g = hld4(nw, ip4);
                        pe[0] *= r * g.x, pe[1] *= r * g.y, pe[2] *= r * g.z, pe[3] *= r * g.w;
                    }
                    const int a0 = low ? j : j - half;
#pragma unroll
                    for (int q = 0; q < 4; ++q) {
                        const float c = cs[a0 + q], sn = cs[half + a0 + q];
                        e[q] = low ? fmaf(e[q], c, -(pe[q] * sn)) : fmaf(e[q], c, pe[q] * sn);
                    }
                }
            }
#pragma unroll
            for (int p2 = 0; p2 < 2; ++p2) {
                const int j = s.rot_half ? -1 : i + 2 * p2 - s.rot_off;
                if (j >= 0 && j < s.rot_dims) {
                    const float c = cs[j >> 1], sn = cs[half + (j >> 1)];
                    const float a0 = e[2 * p2], b0 = e[2 * p2 + 1];
                    e[2 * p2] = fmaf(a0, c, -(b0 * sn));
                    e[2 * p2 + 1] = fmaf(b0, c, a0 * sn);
                }
            }
            if (s.save) *reinterpret_cast<float4*>(s.save + flat + i) = make_float4(e[0], e[1], e[2], e[3]);
            if (s.mix_src) {
                const float4 mv = *reinterpret_cast<const float4*>(s.mix_src + flat + i);
                e[0] = fmaf(s.mix, mv.x - e[0], e[0]), e[1] = fmaf(s.mix, mv.y - e[1], e[1]);
                e[2] = fmaf(s.mix, mv.z - e[2], e[2]), e[3] = fmaf(s.mix, mv.w - e[3], e[3]);
            }
            hst4(dst, i4, make_float4(e[0], e[1], e[2], e[3]));
        }
        return;
    }
    if (s.norm_dims > 0) {
        float ss = 0.f;
#pragma unroll 4
        for (int i = lane; i < s.norm_dims; i += kStep) ss = fmaf(x[i], x[i], ss);
        ss = head_sum(ss);
        r = rsqrtf(ss / static_cast<float>(s.norm_dims) + eps);
    }
    auto normed = [&](int i) -> float {
        float v = x[i];
        if (i < s.norm_dims) v = v * r * hld(nw, i);
        return v;
    };
    for (int i = lane; i < s.width; i += kStep) {
        float v = normed(i);
        const int j = i - s.rot_off;
        if (j >= 0 && j < s.rot_dims) {
            if (s.rot_half) {
                const bool low = j < half;
                const float p = normed(s.rot_off + (low ? j + half : j - half));
                const int a0 = low ? j : j - half;
                const float c = cs[a0], sn = cs[half + a0];
                v = low ? fmaf(v, c, -(p * sn)) : fmaf(v, c, p * sn);
            } else {
                const float p = normed(s.rot_off + (j ^ 1));
                const float c = cs[j >> 1], sn = cs[half + (j >> 1)];
                // pair (u, w) -> (u c - w s, w c + u s)
                v = (j & 1) ? fmaf(v, c, p * sn) : fmaf(v, c, -(p * sn));
            }
        }
        if (s.save) s.save[flat + i] = v;
        if (s.mix_src) v = fmaf(s.mix, s.mix_src[flat + i] - v, v);   // (1 - mix) v + mix m
        hst(dst, i, v);
    }
}

// ---- head preparation behind a short convolution ------------------------------------------------------------------------------
// Per head of a slice: u_t = sum_j w[c][j] x_(t - K + 1 + j) per channel (no bias, no activation; zeros before position 0, the
// K - 1 rows before the step from conv_state [slots, K - 1, C], channel = source column - the first slice's), u written to
// raw_dst's pages as it is (nullable), pairs (2i, 2i + 1) of the first rot_dims elements rotated by the angles at the row's
// position, divided by the root mean square over the head (norm != 0), written to rows or pages. Rows of sequences
// [0, n_inplace) are the only row of their sequence in this step: the warp that read their window writes it back shifted.
struct ConvPrepArgs {
    int n, total_heads, base, C, K, n_inplace;
    atx_conv_head_seg seg[ATX_HEAD_SEGS_MAX];
    const float* src;
    long long ld;
    float* conv_state;
    const int *positions, *slots, *tok_seq, *seq_start, *seq_pos0, *seq_slot;
    int T, bs, rows_per;
    float eps;
};
constexpr int kHeadTaps = 8;

// One warp takes one head and rows_per consecutive rows, the taps' window in registers. A lane owns E elements in groups of VE
// neighbours (VE = min(E, 4)), so a rotated pair lies inside a lane. KT: taps when it is a common number, 0: up to kHeadTaps.
template <typename XT, int E, int KT>
__global__ void __launch_bounds__(256)
conv_head_prepare_kernel(const __grid_constant__ ConvPrepArgs a) {
    constexpr int VE = E < 4 ? E : 4, NG = E / VE;
    constexpr int MT = KT ? KT : kHeadTaps;
    constexpr int NW = MT > 1 ? MT - 1 : 1;
    const int K = KT ? KT : a.K;
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const long long wid = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const long long tile = wid / a.total_heads;
    const int t0 = static_cast<int>(tile) * a.rows_per;
    if (t0 >= a.T) return;
    int hh = static_cast<int>(wid - tile * a.total_heads), si = 0;
    while (si + 1 < a.n && hh >= a.seg[si].heads) {
        hh -= a.seg[si].heads;
        ++si;
    }
    const atx_conv_head_seg& s = a.seg[si];
    const int width = s.width, half = s.rot_dims / 2;
    const long long col = s.src_off + static_cast<long long>(hh) * width;   // source column of the head's first element
    const long long ch = col - a.base;                                     // its channel in the state
    const XT* w = reinterpret_cast<const XT*>(s.w) + static_cast<long long>(hh) * width * K;
    bool on[NG];
    int el[NG];   // first element of each of the lane's groups
    float wt[MT][E];
#pragma unroll
    for (int g = 0; g < NG; ++g) {
        el[g] = g * 32 * VE + lane * VE;
        on[g] = el[g] < width;
#pragma unroll
        for (int e = 0; e < VE; ++e)
#pragma unroll
            for (int j = 0; j < MT; ++j)
                wt[j][g * VE + e] = (on[g] && j < K) ? hld(w, static_cast<long long>(el[g] + e) * K + j) : 0.f;
    }
    pdl_wait();   // the taps are weights: fetched ahead of the wait for the projection
    auto load = [&](const float* p, float (&v)[E]) {   // p: the head's first element of some row
#pragma unroll
        for (int g = 0; g < NG; ++g) {
            if constexpr (VE == 4) {
                const float4 f = on[g] ? *reinterpret_cast<const float4*>(p + el[g]) : make_float4(0.f, 0.f, 0.f, 0.f);
                v[g * VE] = f.x, v[g * VE + 1] = f.y, v[g * VE + 2] = f.z, v[g * VE + 3] = f.w;
            } else {
                const float2 f = on[g] ? *reinterpret_cast<const float2*>(p + el[g]) : make_float2(0.f, 0.f);
                v[g * VE] = f.x, v[g * VE + 1] = f.y;
            }
        }
    };
    auto put = [&](XT* p, const float (&v)[E]) {
#pragma unroll
        for (int g = 0; g < NG; ++g) {
            if (!on[g]) continue;
            if constexpr (VE == 4) {
                hst4(p + el[g], 0, make_float4(v[g * VE], v[g * VE + 1], v[g * VE + 2], v[g * VE + 3]));
            } else if constexpr (sizeof(XT) == 2) {
                *reinterpret_cast<uint32_t*>(p + el[g]) = pack_bf16(v[g * VE], v[g * VE + 1]);
            } else {
                *reinterpret_cast<float2*>(p + el[g]) = make_float2(v[g * VE], v[g * VE + 1]);
            }
        }
    };
    // What the rows of the tile belong to, a row per lane; the angles of a row and its projection are fetched one row ahead.
    int m_seq = -1, m_slot = -1, m_pos = 0;
    if (lane < a.rows_per && t0 + lane < a.T) m_seq = a.tok_seq[t0 + lane], m_slot = a.slots[t0 + lane], m_pos = a.positions[t0 + lane];
    constexpr int NP = E / 2;   // rotated pairs of a lane
    float win[NW][E], cur[E], nxt[E], cn[NP], sn[NP], cx[NP], sx[NP];
    auto angles = [&](int pos) {
        const float* cs = s.rot + static_cast<long long>(pos) * s.rot_dims;
#pragma unroll
        for (int g = 0; g < NG; ++g)
#pragma unroll
            for (int e = 0; e < VE; e += 2) {
                const int p = (el[g] + e) >> 1, q = (g * VE + e) >> 1;
                cx[q] = p < half ? cs[p] : 1.f;
                sx[q] = p < half ? cs[half + p] : 0.f;
            }
    };
    load(a.src + static_cast<long long>(t0) * a.ld + col, nxt);
    if (half > 0) angles(__shfl_sync(0xffffffffu, m_pos, 0));
    int prev_s = -1, prev_i = -2;
    float* st = nullptr;
    for (int r = 0; r < a.rows_per && t0 + r < a.T; ++r) {
        const long long t = t0 + r;
#pragma unroll
        for (int e = 0; e < E; ++e) cur[e] = nxt[e];
#pragma unroll
        for (int q = 0; q < NP; ++q) cn[q] = cx[q], sn[q] = sx[q];
        const int sq = __shfl_sync(0xffffffffu, m_seq, r), slot = __shfl_sync(0xffffffffu, m_slot, r);
        if (r + 1 < a.rows_per && t + 1 < a.T) {
            load(a.src + (t + 1) * a.ld + col, nxt);
            if (half > 0) angles(__shfl_sync(0xffffffffu, m_pos, r + 1));
        }
        if (sq < 0 || slot < 0) {   // padded row
            prev_s = -1;
            continue;
        }
        const int i = sq == prev_s ? prev_i + 1 : static_cast<int>(t) - a.seq_start[sq];   // a sequence's rows are consecutive
        if (sq != prev_s) {
            const int pos0 = a.seq_pos0[sq];
            st = a.conv_state + static_cast<long long>(a.seq_slot[sq]) * (K - 1) * a.C + ch;
#pragma unroll
            for (int j = 0; j < NW; ++j) {
#pragma unroll
                for (int e = 0; e < E; ++e) win[j][e] = 0.f;
                if (j < K - 1) {
                    const int rel = i - (K - 1) + j;   // row of the portion that tap j reads (negative: before it)
                    if (rel >= 0)
                        load(a.src + (t - i + rel) * a.ld + col, win[j]);
                    else if (pos0 + rel >= 0)
                        load(st + static_cast<long long>(K - 1 + rel) * a.C, win[j]);
                }
            }
        }
        float u[E];
#pragma unroll
        for (int e = 0; e < E; ++e) u[e] = 0.f;
#pragma unroll
        for (int j = 0; j < MT; ++j) {
            if (j < K - 1) {
#pragma unroll
                for (int e = 0; e < E; ++e) u[e] = fmaf(wt[j][e], win[j < NW ? j : 0][e], u[e]);
            } else if (j == K - 1) {
#pragma unroll
                for (int e = 0; e < E; ++e) u[e] = fmaf(wt[j][e], cur[e], u[e]);
            }
        }
        // slide: entries 0 .. K - 2 hold the K - 1 inputs before the next row
#pragma unroll
        for (int j = 0; j + 1 < NW; ++j)
            if (j < K - 2)
#pragma unroll
                for (int e = 0; e < E; ++e) win[j][e] = win[j + 1][e];
#pragma unroll
        for (int j = 0; j < NW; ++j)
            if (j == K - 2)
#pragma unroll
                for (int e = 0; e < E; ++e) win[j][e] = cur[e];
        prev_s = sq;
        prev_i = i;
        if (sq < a.n_inplace) {
#pragma unroll
            for (int j = 0; j < NW; ++j) {
                if (j >= K - 1) continue;
                float* p = st + static_cast<long long>(j) * a.C;
#pragma unroll
                for (int g = 0; g < NG; ++g) {
                    if (!on[g]) continue;
                    if constexpr (VE == 4)
                        *reinterpret_cast<float4*>(p + el[g]) = make_float4(win[j][g * VE], win[j][g * VE + 1], win[j][g * VE + 2], win[j][g * VE + 3]);
                    else
                        *reinterpret_cast<float2*>(p + el[g]) = make_float2(win[j][g * VE], win[j][g * VE + 1]);
                }
            }
        }
        const int blk = slot / a.bs, off = slot - blk * a.bs;
        const long long page = ((static_cast<long long>(blk) * s.heads + hh) * a.bs + off) * width;
        if (s.raw_dst) put(reinterpret_cast<XT*>(s.raw_dst) + page, u);
        if (half > 0) {
#pragma unroll
            for (int q = 0; q < NP; ++q) {   // pairs past the rotated range carry the angle 0
                const float x = u[2 * q], y = u[2 * q + 1];
                u[2 * q] = fmaf(x, cn[q], -(y * sn[q]));
                u[2 * q + 1] = fmaf(y, cn[q], x * sn[q]);
            }
        }
        if (s.norm) {
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < E; ++e) ss = fmaf(u[e], u[e], ss);   // elements past the head are zero
            const float rs = rsqrtf(warp_sum(ss) / static_cast<float>(width) + a.eps);
#pragma unroll
            for (int e = 0; e < E; ++e) u[e] *= rs;
        }
        put(reinterpret_cast<XT*>(s.dst) + (s.dst_kind == ATX_HEAD_DST_PAGES ? page : t * s.dst_ld + static_cast<long long>(hh) * width), u);
    }
}

// Any width, alignment and number of taps: a warp per (row, head), the convolved head staged in shared memory.
template <typename XT>
__global__ void __launch_bounds__(256)
conv_head_prepare_any_kernel(const __grid_constant__ ConvPrepArgs a, int stage) {
    extern __shared__ float sconv[];   // [warps][stage]
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    float* u = sconv + (threadIdx.x >> 5) * stage;
    const long long wid = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const long long t = wid / a.total_heads;
    if (t >= a.T) return;
    int hh = static_cast<int>(wid - t * a.total_heads), si = 0;
    while (si + 1 < a.n && hh >= a.seg[si].heads) {
        hh -= a.seg[si].heads;
        ++si;
    }
    const atx_conv_head_seg& s = a.seg[si];
    const int sq = a.tok_seq[t], slot = a.slots[t], K = a.K;
    if (sq < 0 || slot < 0) return;
    const int width = s.width, half = s.rot_dims / 2;
    const long long col = s.src_off + static_cast<long long>(hh) * width, ch = col - a.base;
    const XT* w = reinterpret_cast<const XT*>(s.w) + static_cast<long long>(hh) * width * K;
    const int i = static_cast<int>(t) - a.seq_start[sq], pos0 = a.seq_pos0[sq];
    float* st = a.conv_state + static_cast<long long>(a.seq_slot[sq]) * (K - 1) * a.C + ch;
    const bool inplace = sq < a.n_inplace;
    const int blk = slot / a.bs, off = slot - blk * a.bs;
    const long long page = ((static_cast<long long>(blk) * s.heads + hh) * a.bs + off) * width;
    for (int c = lane; c < width; c += 32) {
        float acc = 0.f;
        for (int j = 0; j < K; ++j) {
            const int rel = i - (K - 1 - j);
            float v = 0.f;
            if (rel >= 0)
                v = a.src[(t - i + rel) * a.ld + col + c];
            else if (pos0 + rel >= 0)
                v = st[static_cast<long long>(K - 1 + rel) * a.C + c];
            if (inplace && j > 0) st[static_cast<long long>(j - 1) * a.C + c] = v;   // entry j - 1 has been read already
            acc = fmaf(hld(w, static_cast<long long>(c) * K + j), v, acc);
        }
        u[c] = acc;
        if (s.raw_dst) hst(reinterpret_cast<XT*>(s.raw_dst) + page, c, acc);
    }
    __syncwarp();
    const float* cs = half > 0 ? s.rot + static_cast<long long>(a.positions[t]) * s.rot_dims : nullptr;
    for (int p = lane; p < half; p += 32) {
        const float c = cs[p], sn = cs[half + p], x = u[2 * p], y = u[2 * p + 1];
        u[2 * p] = fmaf(x, c, -(y * sn));
        u[2 * p + 1] = fmaf(y, c, x * sn);
    }
    __syncwarp();
    float rs = 1.f;
    if (s.norm) {
        float ss = 0.f;
        for (int c = lane; c < width; c += 32) ss = fmaf(u[c], u[c], ss);
        rs = rsqrtf(warp_sum(ss) / static_cast<float>(width) + a.eps);
    }
    XT* dst = reinterpret_cast<XT*>(s.dst) + (s.dst_kind == ATX_HEAD_DST_PAGES ? page : t * s.dst_ld + static_cast<long long>(hh) * width);
    for (int c = lane; c < width; c += 32) hst(dst, c, u[c] * rs);
}

// ---- cap on logits ---------------------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
soft_cap_kernel(float* __restrict__ x, long long ld, int T, int N, float cap) {
    pdl_launch_dependents();
    pdl_wait();
    const long long n = static_cast<long long>(T) * N;
    for (long long e = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; e < n;
         e += static_cast<long long>(gridDim.x) * blockDim.x) {
        const long long t = e / N;
        float* p = x + t * ld + (e - t * N);
        *p = cap * tanhf(*p / cap);
    }
}

// ---- per-head matrix product --------------------------------------------------------------------------------------------
// out[t, h * os + n] = (sum_k X[t, x_off + h * xs + k] W[(h N + n) ldw + k]) (* sigmoid(gate[t, h N + n])).
// FMA pipe, fp32 accumulation in a fixed order; 64 x 64 outputs per CTA, 4 x 4 per thread; blockIdx.z = head.
constexpr int kHM = 64, kHN = 64, kHK = 16;

template <typename XT, typename XI>
__global__ void __launch_bounds__(256)
head_gemm_kernel(const XI* __restrict__ X, long long ldx, int x_off, int xs, const XT* __restrict__ W, long long ldw,
                 const float* __restrict__ gate, long long ldg, XT* __restrict__ out, long long ldo, int o_off, int os,
                 int T, int N, int K) {
    __shared__ float sx[kHK][kHM + 1];
    __shared__ float sw[kHK][kHN + 1];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.z;
    const int t0 = blockIdx.y * kHM, n0 = blockIdx.x * kHN;
    const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
    const XI* Xh = X + x_off + static_cast<long long>(h) * xs;
    const XT* Wh = W + static_cast<long long>(h) * N * ldw;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < K; k0 += kHK) {
        for (int e = threadIdx.x; e < kHM * kHK; e += 256) {
            const int rr = e / kHK, kk = e - rr * kHK;
            const int t = t0 + rr, k = k0 + kk, n = n0 + rr;
            sx[kk][rr] = (t < T && k < K) ? hld(Xh, static_cast<long long>(t) * ldx + k) : 0.f;
            sw[kk][rr] = (n < N && k < K) ? hld(Wh, static_cast<long long>(n) * ldw + k) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < kHK; ++kk) {
            float av[4], bv[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) av[i] = sx[kk][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) bv[j] = sw[kk][tx * 4 + j];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = t0 + ty * 4 + i;
        if (t >= T) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n >= N) continue;
            float v = acc[i][j];
            if (gate) v *= 1.f / (1.f + expf(-gate[static_cast<long long>(t) * ldg + static_cast<long long>(h) * N + n]));
            hst(out, static_cast<long long>(t) * ldo + o_off + static_cast<long long>(h) * os + n, v);
        }
    }
}

// The same product on the tensor cores (bf16 operands, fp32 accumulation): 64 rows x 64 outputs of one head per CTA, a
// warp owns 16 rows; X (fp32 or bf16) and W are staged as bf16 in chunks of 64 reduction elements, zero past the edges.
constexpr int kHT = 64, kHKC = 64, kHLD = kHKC + 8;

template <typename XI>
__global__ void __launch_bounds__(128)
head_gemm_tc_kernel(const XI* __restrict__ X, long long ldx, int x_off, int xs, const __nv_bfloat16* __restrict__ W,
                    long long ldw, const float* __restrict__ gate, long long ldg, __nv_bfloat16* __restrict__ out,
                    long long ldo, int o_off, int os, int T, int N, int K) {
    __shared__ __align__(16) __nv_bfloat16 sx[kHT * kHLD];
    __shared__ __align__(16) __nv_bfloat16 sw[kHT * kHLD];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.z;
    const int t0 = blockIdx.y * kHT, n0 = blockIdx.x * kHT;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const XI* Xh = X + x_off + static_cast<long long>(h) * xs;
    const __nv_bfloat16* Wh = W + static_cast<long long>(h) * N * ldw;
    float acc[kHT / 8][4];
#pragma unroll
    for (int i = 0; i < kHT / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    // eight elements per access where pitches, offsets and K allow it (rows past T or N and columns past K stay zero)
    const bool vec = ((K | x_off | xs) & 7) == 0 && ((ldx | ldw) & 7) == 0 &&
                     ((reinterpret_cast<unsigned long long>(X) | reinterpret_cast<unsigned long long>(W)) & 15) == 0;
    for (int k0 = 0; k0 < K; k0 += kHKC) {
        if (vec) {
            for (int e = threadIdx.x; e < kHT * (kHKC / 8); e += 128) {
                const int r = e / (kHKC / 8), k8 = (e - r * (kHKC / 8)) * 8;
                const int t = t0 + r, n = n0 + r, k = k0 + k8;
                uint4 xv = make_uint4(0, 0, 0, 0), wv = make_uint4(0, 0, 0, 0);
                if (t < T && k < K) {
                    if constexpr (sizeof(XI) == 4) {
                        const float4 a = *reinterpret_cast<const float4*>(Xh + static_cast<long long>(t) * ldx + k);
                        const float4 b = *reinterpret_cast<const float4*>(Xh + static_cast<long long>(t) * ldx + k + 4);
                        xv = make_uint4(pack_bf16(a.x, a.y), pack_bf16(a.z, a.w), pack_bf16(b.x, b.y), pack_bf16(b.z, b.w));
                    } else {
                        xv = *reinterpret_cast<const uint4*>(Xh + static_cast<long long>(t) * ldx + k);
                    }
                }
                if (n < N && k < K) wv = __ldg(reinterpret_cast<const uint4*>(Wh + static_cast<long long>(n) * ldw + k));
                *reinterpret_cast<uint4*>(sx + r * kHLD + k8) = xv;
                *reinterpret_cast<uint4*>(sw + r * kHLD + k8) = wv;
            }
        } else {
            for (int e = threadIdx.x; e < kHT * kHKC; e += 128) {
                const int r = e / kHKC, kk = e - r * kHKC;
                const int t = t0 + r, n = n0 + r, k = k0 + kk;
                const float xv = (t < T && k < K) ? hld(Xh, static_cast<long long>(t) * ldx + k) : 0.f;
                sx[r * kHLD + kk] = __float2bfloat16_rn(xv);
                sw[r * kHLD + kk] = (n < N && k < K) ? Wh[static_cast<long long>(n) * ldw + k] : __float2bfloat16_rn(0.f);
            }
        }
        __syncthreads();
#pragma unroll
        for (int ks = 0; ks < kHKC / 16; ++ks) {
            uint32_t a[4];
            ldsm_x4(smem_u32(sx + (warp * 16 + (lane & 15)) * kHLD + ks * 16 + (lane >> 4) * 8), a[0], a[1], a[2], a[3]);
#pragma unroll
            for (int nb2 = 0; nb2 < kHT / 16; ++nb2) {
                uint32_t b0, b1, b2, b3;
                ldsm_x4(smem_u32(sw + (nb2 * 16 + (lane >> 4) * 8 + (lane & 7)) * kHLD + ks * 16 + ((lane >> 3) & 1) * 8), b0,
                        b1, b2, b3);
                mma_bf16(acc[2 * nb2], a, b0, b1);
                mma_bf16(acc[2 * nb2 + 1], a, b2, b3);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
        const int t = t0 + warp * 16 + (lane >> 2) + 8 * rr;
        if (t >= T) continue;
#pragma unroll
        for (int nb = 0; nb < kHT / 8; ++nb) {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int n = n0 + nb * 8 + (lane & 3) * 2 + e;
                if (n >= N) continue;
                float v = acc[nb][2 * rr + e];
                if (gate) v *= 1.f / (1.f + __expf(-gate[static_cast<long long>(t) * ldg + static_cast<long long>(h) * N + n]));
                out[static_cast<long long>(t) * ldo + o_off + static_cast<long long>(h) * os + n] = __float2bfloat16_rn(v);
            }
        }
    }
}

}  // namespace atx

using namespace atx;

extern "C" {

int atx_tanh_norm(const float* x, const int* rows, float alpha, const void* w, const void* b, void* out, int T, int W,
                  void* zero_ptr, long long zero_bytes, int dtype, int flags, atx_stream_t stream) {
    ATX_REQUIRE(x && w && b && out, "atx_tanh_norm: null pointer");
    ATX_REQUIRE(T > 0 && W > 0, "atx_tanh_norm: bad shape T=%d W=%d", T, W);
    ATX_REQUIRE(zero_bytes >= 0 && zero_bytes % 16 == 0 && (zero_bytes == 0 || zero_ptr),
                "atx_tanh_norm: zero_bytes=%lld must be a non-negative multiple of 16 with a buffer", zero_bytes);
    const long long zv = zero_bytes / 16;
    long long zb = (zv + 256 * 8 - 1) / (256 * 8);
    if (zb > 2048) zb = 2048;
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    cfg.gridDim = dim3(static_cast<unsigned>(T + zb));
    cfg.blockDim = dim3(256);
    cfg.stream = reinterpret_cast<cudaStream_t>(stream);
    set_pdl_attr(cfg, attr, flags);
    ATX_HEADOPS_XT(dtype, ATX_CUDA(cudaLaunchKernelEx(&cfg, tanh_norm_kernel<XT>, x, rows, alpha,
                                                      reinterpret_cast<const XT*>(w), reinterpret_cast<const XT*>(b),
                                                      reinterpret_cast<XT*>(out), T, W,
                                                      reinterpret_cast<uint4*>(zero_ptr), zv)));
    return ATX_OK;
}

int atx_unary_act(const float* in, long long ldi, void* out, long long ldo, int T, int I, int kind, int dtype, int flags,
                  atx_stream_t stream) {
    ATX_REQUIRE(in && out, "atx_unary_act: null pointer");
    ATX_REQUIRE(T > 0 && I > 0 && ldi >= I && ldo >= I, "atx_unary_act: bad shape T=%d I=%d ldi=%lld ldo=%lld", T, I, ldi, ldo);
    ATX_REQUIRE(kind == ATX_ACT_RELU2 || kind == ATX_ACT_GELU_TANH, "atx_unary_act: unknown activation %d", kind);
    const long long n = static_cast<long long>(T) * I;
    long long blocks = (n + 256 * 4 - 1) / (256 * 4);
    if (blocks > 148 * 16) blocks = 148 * 16;
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    cfg.gridDim = dim3(static_cast<unsigned>(blocks));
    cfg.blockDim = dim3(256);
    cfg.stream = reinterpret_cast<cudaStream_t>(stream);
    set_pdl_attr(cfg, attr, flags);
    ATX_HEADOPS_XT(dtype, ATX_CUDA(cudaLaunchKernelEx(&cfg, unary_act_kernel<XT>, in, ldi, reinterpret_cast<XT*>(out), ldo,
                                                      T, I, kind)));
    return ATX_OK;
}

int atx_head_prepare(const float* src, long long ld, const atx_head_seg* segs, int n_segs, const int* positions,
                     const int* slots, int T, int block_size, float eps, int dtype, int flags, atx_stream_t stream) {
    ATX_REQUIRE(src && segs, "atx_head_prepare: null pointer");
    ATX_REQUIRE(T > 0 && n_segs > 0 && n_segs <= ATX_HEAD_SEGS_MAX, "atx_head_prepare: T=%d, %d segments (1..%d)", T,
                n_segs, ATX_HEAD_SEGS_MAX);
    PrepArgs a = {};
    a.n = n_segs;
    for (int i = 0; i < n_segs; ++i) {
        const atx_head_seg& s = segs[i];
        ATX_REQUIRE(s.heads > 0 && s.width > 0 && s.dst && s.src_off >= 0 && s.dst_off >= 0,
                    "atx_head_prepare: segment %d: heads=%d width=%d", i, s.heads, s.width);
        ATX_REQUIRE(s.norm_dims >= 0 && s.norm_dims <= s.width && (s.norm_dims == 0 || s.norm_w),
                    "atx_head_prepare: segment %d: norm over %d of %d elements needs a weight", i, s.norm_dims, s.width);
        ATX_REQUIRE(s.rot_dims >= 0 && s.rot_dims % 2 == 0 && s.rot_off >= 0 && s.rot_off + s.rot_dims <= s.width &&
                        (s.rot_dims == 0 || (s.rot && positions)),
                    "atx_head_prepare: segment %d: rotation of [%d, %d) in a head of %d needs an even count, a table and "
                    "positions", i, s.rot_off, s.rot_off + s.rot_dims, s.width);
        ATX_REQUIRE(s.dst_kind == ATX_HEAD_DST_ROWS || (s.dst_kind == ATX_HEAD_DST_PAGES && slots && block_size > 0),
                    "atx_head_prepare: segment %d: pages need slots and a block size", i);
        a.seg[i] = s;
        a.total_heads += s.heads;
    }
    const long long warps = static_cast<long long>(T) * a.total_heads;
    int widest = 0;
    for (int i = 0; i < n_segs; ++i) widest = segs[i].width > widest ? segs[i].width : widest;
    const bool wide = widest >= 512 && warps <= 1024;   // few, wide heads: a CTA each
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    cfg.gridDim = dim3(static_cast<unsigned>(wide ? warps : (warps + 7) / 8));
    cfg.blockDim = dim3(256);
    cfg.stream = reinterpret_cast<cudaStream_t>(stream);
    set_pdl_attr(cfg, attr, flags);
    if (wide)
        ATX_HEADOPS_XT(dtype, ATX_CUDA(cudaLaunchKernelEx(&cfg, head_prepare_kernel<XT, true>, src, ld, positions, slots, T,
                                                          block_size, eps, a)));
    else
        ATX_HEADOPS_XT(dtype, ATX_CUDA(cudaLaunchKernelEx(&cfg, head_prepare_kernel<XT, false>, src, ld, positions, slots, T,
                                                          block_size, eps, a)));
    return ATX_OK;
}

int atx_conv_head_prepare(const float* src, long long ld, const atx_conv_head_seg* segs, int n_segs, int K, float* conv_state,
                          int C, int n_inplace, const int* positions, const int* slots, const int* tok_seq,
                          const int* seq_start, const int* seq_pos0, const int* seq_slot, int T, int block_size, float eps,
                          int dtype, int flags, atx_stream_t stream) {
    ATX_REQUIRE(src && segs && positions && slots && tok_seq && seq_start && seq_pos0 && seq_slot && (K == 1 || conv_state),
                "atx_conv_head_prepare: null pointer");
    ATX_REQUIRE(T > 0 && n_segs > 0 && n_segs <= ATX_HEAD_SEGS_MAX && K >= 1 && block_size > 0 && n_inplace >= 0,
                "atx_conv_head_prepare: T=%d, %d segments (1..%d), %d taps", T, n_segs, ATX_HEAD_SEGS_MAX, K);
    ConvPrepArgs a = {};
    a.n = n_segs, a.base = segs[0].src_off, a.C = C, a.K = K, a.n_inplace = n_inplace;
    a.src = src, a.ld = ld, a.conv_state = conv_state;
    a.positions = positions, a.slots = slots, a.tok_seq = tok_seq, a.seq_start = seq_start, a.seq_pos0 = seq_pos0, a.seq_slot = seq_slot;
    a.T = T, a.bs = block_size, a.eps = eps;
    auto al16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    int widest = 0, all = 0;   // all: OR of every width, offset and pitch
    bool aligned = al16(src) && al16(conv_state) && ld % 4 == 0 && C % 4 == 0;
    for (int i = 0; i < n_segs; ++i) {
        const atx_conv_head_seg& s = segs[i];
        ATX_REQUIRE(s.heads > 0 && s.width > 0 && s.w && s.dst && s.src_off >= a.base &&
                        s.src_off - a.base + static_cast<long long>(s.heads) * s.width <= C,
                    "atx_conv_head_prepare: segment %d: heads=%d width=%d outside the %d channels", i, s.heads, s.width, C);
        ATX_REQUIRE(s.rot_dims >= 0 && s.rot_dims % 2 == 0 && s.rot_dims <= s.width && (s.rot_dims == 0 || s.rot),
                    "atx_conv_head_prepare: segment %d: rotation of %d of %d elements needs an even count and a table", i, s.rot_dims,
                    s.width);
        ATX_REQUIRE(s.dst_kind == ATX_HEAD_DST_PAGES || (s.dst_kind == ATX_HEAD_DST_ROWS && s.dst_ld >= static_cast<long long>(s.heads) * s.width),
                    "atx_conv_head_prepare: segment %d: bad destination", i);
        a.seg[i] = s;
        a.total_heads += s.heads;
        widest = s.width > widest ? s.width : widest;
        all |= s.width | s.src_off | (s.dst_kind == ATX_HEAD_DST_ROWS ? static_cast<int>(s.dst_ld & 7) : 0);
        aligned = aligned && al16(s.dst) && al16(s.raw_dst);
    }
    const bool fast = aligned && (all & 3) == 0 && widest <= 256 && K <= kHeadTaps;
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    cfg.stream = reinterpret_cast<cudaStream_t>(stream);
    set_pdl_attr(cfg, attr, flags);
    if (fast) {
        a.rows_per = T >= 256 ? 16 : 1;
        const long long warps = static_cast<long long>((T + a.rows_per - 1) / a.rows_per) * a.total_heads;
        const int per = T >= 256 ? 8 : 4;   // decode-sized: smaller CTAs spread over more SMs
        cfg.gridDim = dim3(static_cast<unsigned>((warps + per - 1) / per));
        cfg.blockDim = dim3(32 * per);
#define ATX_CONV_HEADS(E_, KT_) ATX_HEADOPS_XT(dtype, ATX_CUDA(cudaLaunchKernelEx(&cfg, conv_head_prepare_kernel<XT, E_, KT_>, a)))
#define ATX_CONV_HEADS_E(E_)              \
    do {                                  \
        if (K == 4)                       \
            ATX_CONV_HEADS(E_, 4);        \
        else if (K == 3)                  \
            ATX_CONV_HEADS(E_, 3);        \
        else if (K == 2)                  \
            ATX_CONV_HEADS(E_, 2);        \
        else                              \
            ATX_CONV_HEADS(E_, 0);        \
    } while (0)
        if (widest <= 64)
            ATX_CONV_HEADS_E(2);
        else if (widest <= 128)
            ATX_CONV_HEADS_E(4);
        else
            ATX_CONV_HEADS_E(8);
#undef ATX_CONV_HEADS_E
#undef ATX_CONV_HEADS
        return ATX_OK;
    }
    ATX_REQUIRE(widest <= 12000, "atx_conv_head_prepare: heads of %d elements (at most 12000)", widest);
    a.rows_per = 1;
    int per = 12000 / widest;
    per = per > 8 ? 8 : (per < 1 ? 1 : per);
    const long long warps = static_cast<long long>(T) * a.total_heads;
    cfg.gridDim = dim3(static_cast<unsigned>((warps + per - 1) / per));
    cfg.blockDim = dim3(32 * per);
    cfg.dynamicSmemBytes = sizeof(float) * static_cast<size_t>(per) * widest;
    ATX_HEADOPS_XT(dtype, ATX_CUDA(cudaLaunchKernelEx(&cfg, conv_head_prepare_any_kernel<XT>, a, widest)));
    return ATX_OK;
}

int atx_soft_cap(float* x, long long ld, int T, int N, float cap, int flags, atx_stream_t stream) {
    ATX_REQUIRE(x && T > 0 && N > 0 && ld >= N && cap > 0.f, "atx_soft_cap: bad arguments T=%d N=%d ld=%lld cap=%g", T, N, ld, cap);
    const long long n = static_cast<long long>(T) * N;
    long long blocks = (n + 256 * 4 - 1) / (256 * 4);
    if (blocks > 148 * 16) blocks = 148 * 16;
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    cfg.gridDim = dim3(static_cast<unsigned>(blocks));
    cfg.blockDim = dim3(256);
    cfg.stream = reinterpret_cast<cudaStream_t>(stream);
    set_pdl_attr(cfg, attr, flags);
    ATX_CUDA(cudaLaunchKernelEx(&cfg, soft_cap_kernel, x, ld, T, N, cap));
    return ATX_OK;
}

int atx_head_gemm(const void* X, int x_f32, long long ldx, int x_off, int x_head_stride, const void* W, long long ldw,
                  const float* gate, long long ldg, void* out, long long ldo, int o_off, int o_head_stride, int T,
                  int heads, int N, int K, int dtype, int flags, atx_stream_t stream) {
    ATX_REQUIRE(X && W && out, "atx_head_gemm: null pointer");
    ATX_REQUIRE(T > 0 && heads > 0 && heads <= 65535 && N > 0 && K > 0 && ldw >= K,
                "atx_head_gemm: bad shape T=%d heads=%d N=%d K=%d ldw=%lld", T, heads, N, K, ldw);
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr[1];
    cfg.gridDim = dim3((N + kHN - 1) / kHN, (T + kHM - 1) / kHM, heads);
    cfg.blockDim = dim3(256);
    cfg.stream = reinterpret_cast<cudaStream_t>(stream);
    set_pdl_attr(cfg, attr, flags);
    if (dtype == ATX_DT_BF16 && !(flags & ATX_FLAG_HEAD_GEMM_FMA)) {   // bf16: the tensor cores
        using B = __nv_bfloat16;
        cfg.gridDim = dim3((N + kHT - 1) / kHT, (T + kHT - 1) / kHT, heads);
        cfg.blockDim = dim3(128);
        if (x_f32)
            ATX_CUDA(cudaLaunchKernelEx(&cfg, head_gemm_tc_kernel<float>, reinterpret_cast<const float*>(X), ldx, x_off,
                                        x_head_stride, reinterpret_cast<const B*>(W), ldw, gate, ldg,
                                        reinterpret_cast<B*>(out), ldo, o_off, o_head_stride, T, N, K));
        else
            ATX_CUDA(cudaLaunchKernelEx(&cfg, head_gemm_tc_kernel<B>, reinterpret_cast<const B*>(X), ldx, x_off,
                                        x_head_stride, reinterpret_cast<const B*>(W), ldw, gate, ldg,
                                        reinterpret_cast<B*>(out), ldo, o_off, o_head_stride, T, N, K));
        return ATX_OK;
    }
    if (x_f32 || dtype == ATX_DT_F32) {
        ATX_HEADOPS_XT(dtype, ATX_CUDA(cudaLaunchKernelEx(&cfg, head_gemm_kernel<XT, float>,
                                                          reinterpret_cast<const float*>(X), ldx, x_off, x_head_stride,
                                                          reinterpret_cast<const XT*>(W), ldw, gate, ldg,
                                                          reinterpret_cast<XT*>(out), ldo, o_off, o_head_stride, T, N, K)));
    } else {
        using B = __nv_bfloat16;
        ATX_CUDA(cudaLaunchKernelEx(&cfg, head_gemm_kernel<B, B>, reinterpret_cast<const B*>(X), ldx, x_off, x_head_stride,
                                    reinterpret_cast<const B*>(W), ldw, gate, ldg, reinterpret_cast<B*>(out), ldo, o_off,
                                    o_head_stride, T, N, K));
    }
    return ATX_OK;
}

}  // extern "C"
