// Grouped-query attention over a cache of keys and values: query head h reads key / value head h / (heads / kv_heads).  Queries and
// keys are RMS-normed per head and rotated in their first rot_dims dimensions before they meet (the cache holds finished keys);
// a position sees the positions of its own chunk up to itself (chunk = 0: all up to itself); the softmax has a keyless sink
// logit per head; the result is multiplied by sigmoid(gate).  A layer without keys of its own reads the cache of another.
//   grouped_decode_kernel   bf16, few tokens: 8 or 16 query heads of one key / value head against a share of the positions, on the
//                           tensor cores; for a single token per sequence it also makes the queries and the cache row; the last
//                           share to finish adds the others up
//   grouped_rows_kernel     cache rows, and the queries in place (what the kernels below and portions of a few tokens need first)
//   grouped_prefill_kernel  bf16 prompt chunks of one sequence: 64 tokens of a head per CTA
//   grouped_simt_kernel, grouped_combine_kernel   f32 FMA: everything in f32, and shapes the others do not take
// Scores, softmax and sums are f32; on the tensor cores a softmax weight enters the second product as two bf16 terms.
#include <math.h>

#include <algorithm>

#include "stack.cuh"

namespace im {

void grouped_layout(GroupedShape *s, bool own_kv) {
    s->dimP = round_up(s->dim, 8);
    s->vP = round_up(s->vdim, 8);
    s->q_off = 0;
    int at = s->heads * s->dimP;
    s->k_off = s->v_off = -1;
    if (own_kv) {
        s->k_off = at;
        at += s->kv_heads * s->dimP;
        s->v_off = at;
        at += s->kv_heads * s->vP;
    }
    s->g_off = at;
}

namespace {

constexpr float kLog2eGrouped = 1.4426950408889634f;

struct GroupedPlace {
    int slot, pos;
};
__device__ __forceinline__ GroupedPlace grouped_place(const GroupedArgs &a, int m) {
    const int s = m / a.T;
    GroupedPlace p;
    p.slot = a.slot_map ? a.slot_map[s] : s;
    p.pos = a.pos_dev[p.slot] + m % a.T;
    return p;
}
__device__ __forceinline__ int chunk_begin(const GroupedShape &s, int pos) { return s.chunk > 0 ? pos / s.chunk * s.chunk : 0; }

// One head's vector normed, weighted and rotated by a warp; emit(i, value) for every dimension.  src may be what emit writes.
template <typename T, typename F>
__device__ __forceinline__ void norm_rotate(const GroupedArgs &a, const T *src, const float *w, int pos, F emit) {
    const int lane = threadIdx.x & 31, dim = a.s.dim, half = a.s.rot_dims / 2;
    float ss = 0.0f;
    for (int i = lane; i < dim; i += 32) {
        const float v = to_f<T>(src[i]);
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)dim + a.s.eps);
    for (int i = lane; 2 * i < dim; i += 32) {
        float u = to_f<T>(src[2 * i]) * inv * w[2 * i], v = 2 * i + 1 < dim ? to_f<T>(src[2 * i + 1]) * inv * w[2 * i + 1] : 0.0f;
        if (i < half) {
            const float c = a.cosc[(size_t)pos * half + i], s = a.sinc[(size_t)pos * half + i], u0 = u;
            u = u0 * c - v * s;
            v = v * c + u0 * s;
        }
        emit(2 * i, u);
        if (2 * i + 1 < dim) emit(2 * i + 1, v);
    }
}

// Cache rows of one token and key / value head, by a warp
template <typename T>
__device__ __forceinline__ void write_key(const GroupedArgs &a, const T *y, GroupedPlace p, int kvh) {
    T *row = static_cast<T *>(a.kcache) + (((size_t)p.slot * a.s.kv_heads + kvh) * a.max_seq + p.pos) * a.s.dimP;
    norm_rotate<T>(a, y + a.s.k_off + kvh * a.s.dimP, a.k_norm, p.pos, [&](int i, float v) { row[i] = from_f<T>(v); });
}
template <typename T>
__device__ __forceinline__ void write_value(const GroupedArgs &a, const T *y, GroupedPlace p, int kvh) {
    T *row = static_cast<T *>(a.vcache) + (((size_t)p.slot * a.s.kv_heads + kvh) * a.max_seq + p.pos) * a.s.vP;
    const T *src = y + a.s.v_off + kvh * a.s.vP;
    for (int i = threadIdx.x & 31; i < a.s.vdim; i += 32) row[i] = src[i];
}

// grid (tokens, groups of 8 vectors); a warp per vector: query heads, then keys and values if the layer has its own
template <typename T>
__global__ void __launch_bounds__(256) grouped_rows_kernel(const GroupedArgs a) {
    pdl_trigger();
    pdl_wait();
    const int m = blockIdx.x, w = blockIdx.y * 8 + (threadIdx.x >> 5), H = a.s.heads, G = a.s.kv_heads;
    const GroupedPlace p = grouped_place(a, m);
    if (p.pos >= a.max_seq) return;
    T *y = static_cast<T *>(a.y) + (size_t)m * a.ldy;
    if (w < H) {
        T *q = y + a.s.q_off + w * a.s.dimP;
        norm_rotate<T>(a, q, a.q_norm, p.pos, [&](int i, float v) { q[i] = from_f<T>(v); });
    } else if (a.s.k_off >= 0 && w < H + G) {
        write_key<T>(a, y, p, w - H);
    } else if (a.s.k_off >= 0 && w < H + 2 * G) {
        write_value<T>(a, y, p, w - H - G);
    }
}

struct GroupedPart {
    float *po, *pm, *pl;  // [rows][splits][vP], [rows][splits] x 2; row = token * heads + head; maxima in units of log 2
    int splits;
};
// positions [r0, r1) of a share of those that position pos sees; shares are multiples of `unit`
__device__ __forceinline__ void grouped_range(const GroupedArgs &a, int pos, int split, int splits, int unit, int *r0, int *r1) {
    const int lo = chunk_begin(a.s, pos), len = min(pos + 1, a.max_seq) - lo, per = ((len + splits - 1) / splits + unit - 1) / unit * unit;
    *r0 = lo + min(len, split * per);
    *r1 = lo + min(len, split * per + per);
}

// ---- few tokens on the tensor cores ----------------------------------------------------------------------------------------
// grid (kv_heads * head groups, splits, tokens), 4 warps.  Scores are computed transposed: rows are 16 positions, columns 8 query
// heads (NT column tiles), so that all of a product is used from 8 heads a key / value head on.  Every warp walks its own tiles of 16
// positions with its own ring in shared memory, maxima and sums; the four meet at the end.
constexpr int kGdWarps = 4, kGdTile = 16, kGdStages = 3;
constexpr int kGdUnit = kGdWarps * kGdTile;
__host__ __device__ inline int grouped_dimK(const GroupedShape &s) { return (s.dim + 31) / 32 * 32; }
__host__ __device__ inline int grouped_vK(const GroupedShape &s) { return (s.vdim + 15) / 16 * 16; }
inline size_t grouped_decode_smem(const GroupedShape &s, int nt) {
    return (size_t)8 * nt * (grouped_dimK(s) + 8) * 2 + (size_t)kGdWarps * kGdStages * kGdTile * (grouped_dimK(s) + 8 + grouped_vK(s) + 8) * 2;
}

__device__ __forceinline__ unsigned transpose_8x8(unsigned v) {
    unsigned r;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(v));
    return r;
}

// NV: 16-column tiles of the values; FUSED: one token per sequence, queries and the cache row are made here
template <int NV, int NT, bool FUSED>
__global__ void __launch_bounds__(kGdWarps * 32) grouped_decode_kernel(const GroupedArgs a, const GroupedPart part) {
    typedef __nv_bfloat16 T;
    constexpr int NH = 8 * NT;
    extern __shared__ __align__(16) unsigned char grouped_smem[];
    __shared__ float wm[kGdWarps][NH], wl[kGdWarps][NH];
    __shared__ int s_last;
    const GroupedShape &s = a.s;
    const int dimK = grouped_dimK(s), vK = grouped_vK(s), rs = (dimK + 8) * 2, vs = (vK + 8) * 2;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int GQ = s.heads / s.kv_heads, hg = (GQ + NH - 1) / NH, kvh = blockIdx.x / hg, h0 = kvh * GQ + blockIdx.x % hg * NH, nh = min(NH, (kvh + 1) * GQ - h0);
    const int split = blockIdx.y, m = blockIdx.z;
    unsigned char *qs = grouped_smem, *ring = qs + NH * rs + (size_t)warp * kGdStages * kGdTile * (rs + vs);
    pdl_trigger();
    if (!FUSED) pdl_wait();
    // FUSED: positions and older cache rows come from before this step's first kernel (a one-token step is captured with the
    // position update as its last node, and a captured step starts when the one before it has ended)
    const GroupedPlace p = grouped_place(a, m);
    int r0 = 0, r1 = 0;
    if (p.pos < a.max_seq) grouped_range(a, p.pos, split, part.splits, kGdUnit, &r0, &r1);
    const T *kc = static_cast<const T *>(a.kcache) + ((size_t)p.slot * s.kv_heads + kvh) * a.max_seq * s.dimP;
    const T *vc = static_cast<const T *>(a.vcache) + ((size_t)p.slot * s.kv_heads + kvh) * a.max_seq * s.vP;
    const int first = r0 + warp * kGdTile, ntiles = first < r1 ? (r1 - first + kGdUnit - 1) / kGdUnit : 0;
    const int nk = s.dimP / 8, nv = s.vP / 8;
    // padding columns of the ring, once
    for (int i = lane; i < kGdStages * kGdTile * (dimK / 8 - nk); i += 32)
        *reinterpret_cast<uint4 *>(ring + i / (dimK / 8 - nk) * (rs + vs) + (nk + i % (dimK / 8 - nk)) * 16) = make_uint4(0, 0, 0, 0);
    for (int i = lane; i < kGdStages * kGdTile * (vK / 8 - nv); i += 32)
        *reinterpret_cast<uint4 *>(ring + i / (vK / 8 - nv) * (rs + vs) + rs + (nv + i % (vK / 8 - nv)) * 16) = make_uint4(0, 0, 0, 0);
    // a lane copies the 16-byte vectors lc, lc + 32, ... of the rows lr, lr + rows, ... ([key | value] of a position is one row)
    const int per = nk + nv, rows = per <= 32 ? 32 / per : 1, lr = per <= 32 ? lane / per : 0, lc = per <= 32 ? lane % per : lane;
    auto issue = [&](int it) {
        if (it < ntiles && lr < rows) {
            const int p0 = first + it * kGdUnit;
            unsigned char *dst = ring + it % kGdStages * kGdTile * (rs + vs) + lr * (rs + vs);
            for (int c = lc; c < per; c += per <= 32 ? per : 32) {
                const T *src = c < nk ? kc + c * 8 : vc + (c - nk) * 8;
                const int stride = c < nk ? s.dimP : s.vP;
                unsigned char *d = dst + (c < nk ? c * 16 : rs + (c - nk) * 16);
#pragma unroll 4
                for (int r = lr; r < kGdTile; r += rows, d += rows * (rs + vs)) cp_async16(d, src + (size_t)min(p0 + r, r1 - 1) * stride);
            }
        }
        cp_async_commit();
    };
    int issued = 0;
    if (FUSED) {
        while (issued < kGdStages - 1 && first + issued * kGdUnit + kGdTile <= p.pos) issue(issued++);
        pdl_wait();
    }
    const T *y = static_cast<const T *>(a.y) + (size_t)m * a.ldy;
    if (FUSED && s.k_off >= 0 && r1 > r0 && r1 == p.pos + 1) {  // the share with the token's own position
        if (warp == 0) write_key<T>(a, y, p, kvh);
        if (warp == 1) write_value<T>(a, y, p, kvh);
        __threadfence();  // the copies below read it back past the first-level cache
    }
    for (int h = warp; h < NH; h += kGdWarps) {
        T *q = reinterpret_cast<T *>(qs + h * rs);
        const bool live = h < nh && p.pos < a.max_seq;
        for (int i = (live ? s.dim : 0) + lane; i < dimK; i += 32) q[i] = from_f<T>(0.0f);
        if (!live) continue;
        const T *src = y + s.q_off + (h0 + h) * s.dimP;
        if (FUSED) norm_rotate<T>(a, src, a.q_norm, p.pos, [&](int i, float v) { q[i] = from_f<T>(v); });
        else
            for (int i = lane; i < s.dim; i += 32) q[i] = src[i];
    }
    __syncthreads();
    while (issued < kGdStages - 1) issue(issued++);
    const float scale2 = s.scale * kLog2eGrouped;
    float m_run[NT][2], l_run[NT][2], o[NV][NT][4];
#pragma unroll
    for (int j = 0; j < NT; j++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            m_run[j][e] = -INFINITY;
            l_run[j][e] = 0.0f;
        }
#pragma unroll
    for (int i = 0; i < NV; i++)
#pragma unroll
        for (int j = 0; j < NT; j++) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.0f;
    const unsigned rbase = (unsigned)__cvta_generic_to_shared(ring), qbase = (unsigned)__cvta_generic_to_shared(qs) + (lane & 7) * rs + (lane >> 3) * 16;
    const unsigned kl = (lane & 15) * (rs + vs) + (lane >> 4) * 16, vl = ((lane >> 4) * 8 + (lane & 7)) * (rs + vs) + rs + ((lane >> 3) & 1) * 16;
    for (int it = 0; it < ntiles; it++) {
        cp_async_wait<kGdStages - 2>();
        __syncwarp();
        issue(it + kGdStages - 1);  // into the stage that the tile before this one used
        const unsigned st = rbase + it % kGdStages * kGdTile * (rs + vs);
        const int p0 = first + it * kGdUnit;
        float sc[NT][4];
#pragma unroll
        for (int j = 0; j < NT; j++) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.0f;
#pragma unroll 4
        for (int kk = 0; kk < dimK / 32; kk++) {
            unsigned k0[4], k1[4];
            ldsm_x4(k0, st + kl + kk * 64);
            ldsm_x4(k1, st + kl + kk * 64 + 32);
#pragma unroll
            for (int j = 0; j < NT; j++) {
                unsigned b[4];
                ldsm_x4(b, qbase + j * 8 * rs + kk * 64);
                mma_bf16(sc[j], k0[0], k0[1], k0[2], k0[3], b[0], b[1]);
                mma_bf16(sc[j], k1[0], k1[1], k1[2], k1[3], b[2], b[3]);
            }
        }
        unsigned hi[NT][2], lo[NT][2];
        bool moved = false;
        float corr[NT][2];
#pragma unroll
        for (int j = 0; j < NT; j++) {
#pragma unroll
            for (int e = 0; e < 4; e++) sc[j][e] = p0 + g + 8 * (e >> 1) < r1 ? sc[j][e] * scale2 : -INFINITY;
#pragma unroll
            for (int e = 0; e < 2; e++) {
                float mx = fmaxf(sc[j][e], sc[j][2 + e]);
#pragma unroll
                for (int x = 4; x < 32; x *= 2) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
                const float m_new = fmaxf(m_run[j][e], mx);  // finite: every tile has a position
                moved |= m_new > m_run[j][e];
                corr[j][e] = exp2f(m_run[j][e] - m_new);
                m_run[j][e] = m_new;
                sc[j][e] = exp2f(sc[j][e] - m_new);
                sc[j][2 + e] = exp2f(sc[j][2 + e] - m_new);
                l_run[j][e] = l_run[j][e] * corr[j][e] + sc[j][e] + sc[j][2 + e];
            }
#pragma unroll
            for (int r = 0; r < 2; r++) {
                unsigned terms[2];
                split_bf2<2>(sc[j][2 * r], sc[j][2 * r + 1], terms);
                hi[j][r] = transpose_8x8(terms[0]);
                lo[j][r] = transpose_8x8(terms[1]);
            }
        }
        if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
            for (int i = 0; i < NV; i++)
#pragma unroll
                for (int j = 0; j < NT; j++) {
                    o[i][j][0] *= corr[j][0]; o[i][j][1] *= corr[j][1];
                    o[i][j][2] *= corr[j][0]; o[i][j][3] *= corr[j][1];
                }
        }
#pragma unroll
        for (int i = 0; i < NV; i++)
            if (i * 16 < vK) {
                unsigned v[4];
                ldsm_x4_t(v, st + vl + i * 32);
#pragma unroll
                for (int j = 0; j < NT; j++) {
                    mma_bf16(o[i][j], v[0], v[1], v[2], v[3], hi[j][0], hi[j][1]);
                    mma_bf16(o[i][j], v[0], v[1], v[2], v[3], lo[j][0], lo[j][1]);
                }
            }
    }
    cp_async_wait<0>();
    // the four warps' maxima, sums and outputs; the outputs [warp][head][vK] take the ring's place
#pragma unroll
    for (int j = 0; j < NT; j++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            float l = l_run[j][e];
#pragma unroll
            for (int x = 4; x < 32; x *= 2) l += __shfl_xor_sync(0xffffffffu, l, x);
            if (g == 0) {
                wm[warp][j * 8 + 2 * t + e] = m_run[j][e];
                wl[warp][j * 8 + 2 * t + e] = l;
            }
        }
    __syncthreads();
    float *ow = reinterpret_cast<float *>(qs + NH * rs);
#pragma unroll
    for (int i = 0; i < NV; i++)
        if (i * 16 < vK)
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) ow[((size_t)warp * NH + j * 8 + 2 * t + (e & 1)) * vK + i * 16 + g + 8 * (e >> 1)] = o[i][j][e];
    __syncthreads();
    const size_t row0 = (size_t)m * s.heads + h0;
    const T *gate = y + s.g_off + h0 * s.vP;
    T *out = static_cast<T *>(a.out) + (size_t)m * a.ldo + h0 * s.vP;
    for (int i = tid; i < nh * s.vP; i += kGdWarps * 32) {
        const int h = i / s.vP, v = i % s.vP;
        const float sink = a.sink[h0 + h] * kLog2eGrouped;
        float mx = part.splits == 1 ? sink : -INFINITY;
#pragma unroll
        for (int w = 0; w < kGdWarps; w++) mx = fmaxf(mx, wm[w][h]);
        float sum = 0.0f, l = part.splits == 1 ? exp2f(sink - mx) : 0.0f;
#pragma unroll
        for (int w = 0; w < kGdWarps; w++)
            if (wm[w][h] != -INFINITY) {
                const float f = exp2f(wm[w][h] - mx);
                sum = fmaf(f, ow[((size_t)w * NH + h) * vK + v], sum);
                l = fmaf(f, wl[w][h], l);
            }
        if (part.splits == 1) {
            out[i] = from_f<T>(sum / l * sigmoid_f(to_f<T>(gate[i])));
        } else {
            part.po[((row0 + h) * part.splits + split) * s.vP + v] = sum;
            if (v == 0) {
                part.pm[(row0 + h) * part.splits + split] = mx;
                part.pl[(row0 + h) * part.splits + split] = l;
            }
        }
    }
    if (part.splits == 1) return;
    // the last share to arrive adds them up
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        unsigned *c = a.counters + (size_t)m * gridDim.x + blockIdx.x;
        s_last = atomicAdd(c, 1u) == gridDim.y - 1;
        if (s_last) *c = 0;
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    float *wk = reinterpret_cast<float *>(qs + NH * rs);  // [head][splits]: weight of a share in the normalised sum
    for (int h = warp; h < nh; h += kGdWarps) {
        const bool live = lane < part.splits;
        const float mk = live ? __ldcg(part.pm + (row0 + h) * part.splits + lane) : -INFINITY, lk = live ? __ldcg(part.pl + (row0 + h) * part.splits + lane) : 0.0f;
        const float sink = a.sink[h0 + h] * kLog2eGrouped, mx = fmaxf(sink, warp_max(mk));
        const float f = mk == -INFINITY ? 0.0f : exp2f(mk - mx), l = warp_sum(f * lk) + exp2f(sink - mx);
        if (live) wk[h * part.splits + lane] = f / l;
    }
    __syncthreads();
    for (int i = tid; i < nh * s.vP; i += kGdWarps * 32) {
        const int h = i / s.vP, v = i % s.vP;
        const float *src = part.po + (row0 + h) * part.splits * s.vP + v;
        float sum = 0.0f;
#pragma unroll 8
        for (int k = 0; k < part.splits; k++) sum = fmaf(wk[h * part.splits + k], __ldcg(src + (size_t)k * s.vP), sum);
        out[i] = from_f<T>(sum * sigmoid_f(to_f<T>(gate[i])));
    }
}

// ---- prompt chunks of one sequence -----------------------------------------------------------------------------------------
// grid (ceil(T / 64), heads), 4 warps of 16 tokens, tiles of 32 positions, two in flight.
constexpr int kGpM = 64, kGpN = 32, kGpThreads = kGpM * 2, kGpNB = kGpN / 8;
inline size_t grouped_prefill_smem(const GroupedShape &s, int dv) {
    return (size_t)(kGpM + 2 * kGpN) * (grouped_dimK(s) + 8) * 2 + (size_t)2 * kGpN * (dv + 8) * 2;
}

template <int DV>  // value columns, padded
__global__ void __launch_bounds__(kGpThreads, DV <= 128 ? 3 : 1) grouped_prefill_kernel(const GroupedArgs a) {
    typedef __nv_bfloat16 T;
    constexpr int NTH = kGpThreads, ND = DV / 8;
    extern __shared__ __align__(16) unsigned char grouped_smem[];
    const GroupedShape &s = a.s;
    const int qk = grouped_dimK(s), rs = (qk + 8) * 2, vs = (DV + 8) * 2;
    unsigned char *qs = grouped_smem, *kt = qs + kGpM * rs, *vt = kt + 2 * kGpN * rs;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int tb = gridDim.x - 1 - blockIdx.x, h = blockIdx.y, kvh = h / (s.heads / s.kv_heads);  // latest (longest) blocks first
    pdl_trigger();
    const int P = a.host_pos, nq = s.dimP / 8, nvv = s.vP / 8;
    // padding columns once; everything else is overwritten by the copies
    for (int i = tid; i < (kGpM + 2 * kGpN) * (qk / 8); i += NTH)
        if (i % (qk / 8) >= nq) *reinterpret_cast<uint4 *>(qs + (size_t)(i / (qk / 8)) * rs + (i % (qk / 8)) * 16) = make_uint4(0, 0, 0, 0);
    for (int i = tid; i < 2 * kGpN * (DV / 8); i += NTH)
        if (i % (DV / 8) >= nvv) *reinterpret_cast<uint4 *>(vt + (size_t)(i / (DV / 8)) * vs + (i % (DV / 8)) * 16) = make_uint4(0, 0, 0, 0);
    pdl_wait();
    const T *kc = static_cast<const T *>(a.kcache) + ((size_t)a.host_slot * s.kv_heads + kvh) * a.max_seq * s.dimP;
    const T *vc = static_cast<const T *>(a.vcache) + ((size_t)a.host_slot * s.kv_heads + kvh) * a.max_seq * s.vP;
    const T *q = static_cast<const T *>(a.y) + s.q_off + (size_t)h * s.dimP;
    for (int i = tid; i < kGpM * nq; i += NTH) {
        const int r = i / nq, c = i % nq, tok = tb * kGpM + r;
        *reinterpret_cast<uint4 *>(qs + r * rs + c * 16) = tok < a.T ? *reinterpret_cast<const uint4 *>(q + (size_t)tok * a.ldy + c * 8) : make_uint4(0, 0, 0, 0);
    }
    const int n_begin = chunk_begin(s, P + tb * kGpM), n_end = P + min(tb * kGpM + kGpM, a.T), ntiles = (n_end - n_begin + kGpN - 1) / kGpN;
    auto load_tile = [&](int buf, int p0) {
        unsigned char *kd = kt + (size_t)buf * kGpN * rs, *vd = vt + (size_t)buf * kGpN * vs;
        for (int r = warp; r < kGpN; r += NTH / 32) {
            const size_t p = (size_t)min(p0 + r, n_end - 1);
            for (int c = lane; c < nq + nvv; c += 32) {
                if (c < nq) cp_async16(kd + r * rs + c * 16, kc + p * s.dimP + c * 8);
                else cp_async16(vd + r * vs + (c - nq) * 16, vc + p * s.vP + (c - nq) * 8);
            }
        }
        cp_async_commit();
    };
    load_tile(0, n_begin);
    // positions that each of this thread's two rows, any row and every row of the warp see
    const int tok0 = tb * kGpM + warp * 16 + g, w0 = tb * kGpM + warp * 16;
    int from[2], lim[2];
#pragma unroll
    for (int r = 0; r < 2; r++) {
        lim[r] = tok0 + 8 * r < a.T ? P + tok0 + 8 * r : -1;
        from[r] = lim[r] < 0 ? 0 : chunk_begin(s, lim[r]);
    }
    const int warp_begin = chunk_begin(s, P + w0), warp_end = w0 < a.T ? P + min(w0 + 16, a.T) : 0;
    const bool whole = w0 + 16 <= a.T;
    const int full_begin = chunk_begin(s, P + w0 + 15), full_end = whole ? P + w0 + 1 : 0;
    const float scale2 = s.scale * kLog2eGrouped;  // scores in units of log 2: one exponential instruction each
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
    float o[ND][4];
#pragma unroll
    for (int i = 0; i < ND; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const unsigned qa = (unsigned)__cvta_generic_to_shared(qs) + (warp * 16 + (lane & 15)) * rs + (lane >> 4) * 16;
    const unsigned ka = (unsigned)__cvta_generic_to_shared(kt) + (lane & 7) * rs + (lane >> 3) * 16;
    const unsigned va = (unsigned)__cvta_generic_to_shared(vt) + (lane & 15) * vs + (lane >> 4) * 16;
    for (int it = 0; it < ntiles; it++) {
        const int buf = it & 1, p0 = n_begin + it * kGpN;
        if (it + 1 < ntiles) {
            load_tile(buf ^ 1, p0 + kGpN);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        if (p0 < warp_end && p0 + kGpN > warp_begin) {
            float sc[kGpNB][4];
#pragma unroll
            for (int nb = 0; nb < kGpNB; nb++) sc[nb][0] = sc[nb][1] = sc[nb][2] = sc[nb][3] = 0.0f;
#pragma unroll 2
            for (int kk = 0; kk < qk / 32; kk++) {
                unsigned a0[4], a1[4];
                ldsm_x4(a0, qa + kk * 64);
                ldsm_x4(a1, qa + kk * 64 + 32);
#pragma unroll
                for (int nb = 0; nb < kGpNB; nb++) {
                    unsigned b[4];
                    ldsm_x4(b, ka + (buf * kGpN + 8 * nb) * rs + kk * 64);
                    mma_bf16(sc[nb], a0[0], a0[1], a0[2], a0[3], b[0], b[1]);
                    mma_bf16(sc[nb], a1[0], a1[1], a1[2], a1[3], b[2], b[3]);
                }
            }
            float corr[2], mx[2] = {-INFINITY, -INFINITY};
            if (p0 >= full_begin && p0 + kGpN <= full_end) {
#pragma unroll
                for (int nb = 0; nb < kGpNB; nb++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        sc[nb][e] *= scale2;
                        mx[e >> 1] = fmaxf(mx[e >> 1], sc[nb][e]);
                    }
            } else {
#pragma unroll
                for (int nb = 0; nb < kGpNB; nb++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int p = p0 + 8 * nb + 2 * t + (e & 1);
                        sc[nb][e] = p >= from[e >> 1] && p <= lim[e >> 1] ? sc[nb][e] * scale2 : -INFINITY;
                        mx[e >> 1] = fmaxf(mx[e >> 1], sc[nb][e]);
                    }
            }
            bool moved = false;
#pragma unroll
            for (int r = 0; r < 2; r++) {
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
                const float m_new = fmaxf(m_run[r], mx[r]);
                moved |= m_new > m_run[r];
                corr[r] = m_new == -INFINITY ? 1.0f : exp2f(m_run[r] - m_new);
                m_run[r] = m_new;
                l_run[r] *= corr[r];
            }
            if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
                for (int i = 0; i < ND; i++) {
                    o[i][0] *= corr[0]; o[i][1] *= corr[0];
                    o[i][2] *= corr[1]; o[i][3] *= corr[1];
                }
            }
            const float base[2] = {m_run[0] == -INFINITY ? 0.0f : m_run[0], m_run[1] == -INFINITY ? 0.0f : m_run[1]};
#pragma unroll
            for (int kb = 0; kb < kGpN / 16; kb++) {
                unsigned hi[4], lo[4];
#pragma unroll
                for (int hb = 0; hb < 2; hb++)
#pragma unroll
                    for (int r = 0; r < 2; r++) {
                        const float x0 = exp2f(sc[2 * kb + hb][2 * r] - base[r]), x1 = exp2f(sc[2 * kb + hb][2 * r + 1] - base[r]);  // a masked score gives zero
                        l_run[r] += x0 + x1;
                        unsigned terms[2];
                        split_bf2<2>(x0, x1, terms);
                        hi[2 * hb + r] = terms[0];
                        lo[2 * hb + r] = terms[1];
                    }
#pragma unroll
                for (int nd = 0; nd < ND; nd += 2) {
                    if (DV > 64 && nd * 8 >= s.vP) break;
                    unsigned b[4];
                    ldsm_x4_t(b, va + (buf * kGpN + 16 * kb) * vs + nd * 16);
                    mma_bf16(o[nd], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
                    mma_bf16(o[nd + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
                    mma_bf16(o[nd], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
                    mma_bf16(o[nd + 1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
                }
            }
        }
        __syncthreads();
    }
    const float sink = a.sink[h] * kLog2eGrouped;
#pragma unroll
    for (int r = 0; r < 2; r++) {
        float l = l_run[r];
        l += __shfl_xor_sync(0xffffffffu, l, 1);
        l += __shfl_xor_sync(0xffffffffu, l, 2);
        const int tok = tok0 + 8 * r;
        if (tok < a.T) {
            const float gm = fmaxf(m_run[r], sink), c = exp2f(m_run[r] - gm), inv = c / (l * c + exp2f(sink - gm));
            const T *gate = static_cast<const T *>(a.y) + (size_t)tok * a.ldy + s.g_off + h * s.vP;
            T *dst = static_cast<T *>(a.out) + (size_t)tok * a.ldo + h * s.vP;
#pragma unroll
            for (int nd = 0; nd < ND; nd++) {
                const int c2 = 8 * nd + 2 * t;
                if (c2 < s.vP) {
                    const unsigned z = *reinterpret_cast<const unsigned *>(gate + c2);
                    *reinterpret_cast<unsigned *>(dst + c2) = pack_bf2(o[nd][2 * r] * inv * sigmoid_f(__uint_as_float(z << 16)),
                                                                       o[nd][2 * r + 1] * inv * sigmoid_f(__uint_as_float(z & 0xffff0000u)));
                }
            }
        }
    }
}

// ---- f32 FMA -----------------------------------------------------------------------------------------------------------------
// grid (heads, splits, tokens), 4 warps; tiles of 128 positions: a warp per position for the scores, a thread per value column
// (up to 8 of them) for the weighted sum.
constexpr int kGsThreads = 128, kGsTile = 128, kGsCols = 8;
template <typename T>
__global__ void __launch_bounds__(kGsThreads) grouped_simt_kernel(const GroupedArgs a, const GroupedPart part) {
    constexpr int V = Vec16<T>::n;
    extern __shared__ __align__(16) unsigned char grouped_smem[];
    float *qs = reinterpret_cast<float *>(grouped_smem), *w = qs + a.s.dimP;
    __shared__ float sh[32];
    const GroupedShape &s = a.s;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, split = blockIdx.y, mtok = blockIdx.z, kvh = h / (s.heads / s.kv_heads);
    pdl_trigger();
    pdl_wait();
    const GroupedPlace p = grouped_place(a, mtok);
    int r0 = 0, r1 = 0;
    if (p.pos < a.max_seq) grouped_range(a, p.pos, split, part.splits, kGsTile, &r0, &r1);
    const size_t row = (size_t)mtok * s.heads + h;
    const T *kc = static_cast<const T *>(a.kcache) + ((size_t)p.slot * s.kv_heads + kvh) * a.max_seq * s.dimP;
    const T *vc = static_cast<const T *>(a.vcache) + ((size_t)p.slot * s.kv_heads + kvh) * a.max_seq * s.vP;
    const T *q = static_cast<const T *>(a.y) + (size_t)mtok * a.ldy + s.q_off + h * s.dimP;
    for (int i = tid; i < s.dimP; i += kGsThreads) qs[i] = to_f<T>(q[i]);
    float m = -INFINITY, l = 0.0f, acc[kGsCols];
#pragma unroll
    for (int c = 0; c < kGsCols; c++) acc[c] = 0.0f;
    for (int p0 = r0; p0 < r1; p0 += kGsTile) {
        __syncthreads();
        const int n = min(kGsTile, r1 - p0);
        for (int j = warp; j < n; j += kGsThreads / 32) {
            const uint4 *kr = reinterpret_cast<const uint4 *>(kc + (size_t)(p0 + j) * s.dimP);
            float dot = 0.0f;
            for (int i = lane; i < s.dimP / V; i += 32) {
                float k[V];
                Vec16<T>::unpack(kr[i], k);
#pragma unroll
                for (int e = 0; e < V; e++) dot = fmaf(qs[i * V + e], k[e], dot);
            }
            dot = warp_sum(dot);
            if (lane == 0) w[j] = dot * s.scale;
        }
        __syncthreads();
        const float sv = tid < n ? w[tid] : -INFINITY;
        float mx = warp_max(sv);
        if (lane == 0) sh[warp] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(sh[0], sh[1]), fmaxf(sh[2], sh[3]));
        const float m_new = fmaxf(m, mx), corr = expf(m - m_new);
        m = m_new;
        const float e = tid < n ? expf(sv - m) : 0.0f;
        w[tid] = e;
        l = l * corr + block_sum_f(e, sh);
#pragma unroll
        for (int c = 0; c < kGsCols; c++) acc[c] *= corr;
        for (int j = 0; j < n; j++) {
            const T *vr = vc + (size_t)(p0 + j) * s.vP;
            const float wj = w[j];
#pragma unroll
            for (int c = 0; c < kGsCols; c++)
                if (tid + c * kGsThreads < s.vP) acc[c] = fmaf(wj, to_f<T>(vr[tid + c * kGsThreads]), acc[c]);
        }
    }
#pragma unroll
    for (int c = 0; c < kGsCols; c++)
        if (tid + c * kGsThreads < s.vP) part.po[(row * part.splits + split) * s.vP + tid + c * kGsThreads] = acc[c];
    if (tid == 0) {
        part.pm[row * part.splits + split] = m;
        part.pl[row * part.splits + split] = l;
    }
}

// grid (tokens * heads): shares, sink and gate
template <typename T>
__global__ void __launch_bounds__(kGsThreads) grouped_combine_kernel(const GroupedArgs a, const GroupedPart p) {
    pdl_trigger();
    pdl_wait();
    const GroupedShape &s = a.s;
    const size_t row = blockIdx.x;
    const int m = blockIdx.x / s.heads, h = blockIdx.x % s.heads;
    float gm = a.sink[h];
    for (int k = 0; k < p.splits; k++) gm = fmaxf(gm, p.pm[row * p.splits + k]);
    float l = expf(a.sink[h] - gm);
    for (int k = 0; k < p.splits; k++) l += p.pl[row * p.splits + k] * expf(p.pm[row * p.splits + k] - gm);
    const T *gate = static_cast<const T *>(a.y) + (size_t)m * a.ldy + s.g_off + h * s.vP;
    T *out = static_cast<T *>(a.out) + (size_t)m * a.ldo + h * s.vP;
    for (int v = threadIdx.x; v < s.vP; v += kGsThreads) {
        float sum = 0.0f;
        for (int k = 0; k < p.splits; k++) sum += p.po[(row * p.splits + k) * s.vP + v] * expf(p.pm[row * p.splits + k] - gm);
        out[v] = from_f<T>(sum / l * sigmoid_f(to_f<T>(gate[v])));
    }
}

// ---- host ---------------------------------------------------------------------------------------------------------------
constexpr size_t kGroupedSmemMax = 220 * 1024;
constexpr int kGroupedSplits = 32;  // a warp adds up the shares of a head
int head_tiles(const GroupedShape &s) { return s.heads / s.kv_heads > 8 ? 2 : 1; }
int head_groups(const GroupedShape &s) {
    const int gq = s.heads / s.kv_heads, nh = 8 * head_tiles(s);
    return (gq + nh - 1) / nh;
}
bool decode_tc(const GroupedShape &s) { return s.vP <= 256 && grouped_decode_smem(s, head_tiles(s)) <= kGroupedSmemMax; }
int prefill_dv(const GroupedShape &s) { return s.vP <= 64 ? 64 : s.vP <= 128 ? 128 : s.vP <= 256 ? 256 : 0; }
int auto_splits(const Device *dev, const GroupedShape &s, int f32, int tokens, int ctx) {
    const bool tc = !f32 && decode_tc(s);
    const int ctas = tokens * (tc ? s.kv_heads * head_groups(s) : s.heads), unit = tc ? kGdUnit : kGsTile;
    const int seen = s.chunk > 0 ? std::min(s.chunk, ctx) : ctx;
    const int n = std::min((tc ? 2 : 4) * dev->sm_count / ctas, (seen + unit - 1) / unit);
    return std::max(1, std::min(n, kGroupedSplits));
}
size_t part_bytes_for(const GroupedShape &s, size_t rows, int splits) { return rows * (size_t)splits * (s.vP + 2) * sizeof(float); }

template <int NV, int NT>
int decode_launch(const GroupedArgs &a, const GroupedPart &p, cudaStream_t st) {
    const dim3 grid(a.s.kv_heads * head_groups(a.s), p.splits, a.nseq * a.T), block(kGdWarps * 32);
    const size_t smem = grouped_decode_smem(a.s, NT);
    if (a.T == 1) IM_CUDA_CHECK(launch_k(grouped_decode_kernel<NV, NT, true>, grid, block, smem, st, a, p));
    else IM_CUDA_CHECK(launch_k(grouped_decode_kernel<NV, NT, false>, grid, block, smem, st, a, p));
    return IM_OK;
}
template <int NT>
int decode_any(const GroupedArgs &a, const GroupedPart &p, cudaStream_t st) {
    if (a.s.vP <= 64) return decode_launch<4, NT>(a, p, st);
    if (a.s.vP <= 128) return decode_launch<8, NT>(a, p, st);
    return decode_launch<16, NT>(a, p, st);
}
template <typename T>
int rows_launch(const GroupedArgs &a, cudaStream_t st) {
    const int n = a.s.heads + (a.s.k_off >= 0 ? 2 * a.s.kv_heads : 0);
    IM_CUDA_CHECK(launch_k(grouped_rows_kernel<T>, dim3(a.nseq * a.T, (n + 7) / 8), dim3(256), 0, st, a));
    return IM_OK;
}
template <int DV>
int prefill_launch(const GroupedArgs &a, cudaStream_t st) {
    IM_CUDA_CHECK(launch_k(grouped_prefill_kernel<DV>, dim3((a.T + kGpM - 1) / kGpM, a.s.heads), dim3(kGpThreads), grouped_prefill_smem(a.s, DV), st, a));
    return IM_OK;
}
template <typename T>
int simt_launch(const GroupedArgs &a, const GroupedPart &p, cudaStream_t st) {
    const int M = a.nseq * a.T;
    IM_CUDA_CHECK(launch_k(grouped_simt_kernel<T>, dim3(a.s.heads, p.splits, M), dim3(kGsThreads), (size_t)(a.s.dimP + kGsTile) * sizeof(float), st, a, p));
    IM_CUDA_CHECK(launch_k(grouped_combine_kernel<T>, dim3(M * a.s.heads), dim3(kGsThreads), 0, st, a, p));
    return IM_OK;
}

}  // namespace

bool grouped_prefills(const GroupedShape &s) { return prefill_dv(s) > 0 && grouped_prefill_smem(s, prefill_dv(s)) <= kGroupedSmemMax; }

int grouped_prepare(const Device *dev) {
    static DeviceOnce once;
    if (!once.first(dev->ordinal)) return IM_OK;
    const int mx = (int)kGroupedSmemMax;
#define IM_SMEM(k) IM_CUDA_CHECK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, mx))
    IM_SMEM((grouped_decode_kernel<4, 1, true>)); IM_SMEM((grouped_decode_kernel<8, 1, true>)); IM_SMEM((grouped_decode_kernel<16, 1, true>));
    IM_SMEM((grouped_decode_kernel<4, 2, true>)); IM_SMEM((grouped_decode_kernel<8, 2, true>)); IM_SMEM((grouped_decode_kernel<16, 2, true>));
    IM_SMEM((grouped_decode_kernel<4, 1, false>)); IM_SMEM((grouped_decode_kernel<8, 1, false>)); IM_SMEM((grouped_decode_kernel<16, 1, false>));
    IM_SMEM((grouped_decode_kernel<4, 2, false>)); IM_SMEM((grouped_decode_kernel<8, 2, false>)); IM_SMEM((grouped_decode_kernel<16, 2, false>));
    IM_SMEM(grouped_prefill_kernel<64>); IM_SMEM(grouped_prefill_kernel<128>); IM_SMEM(grouped_prefill_kernel<256>);
#undef IM_SMEM
    return IM_OK;
}

// Scratch for the partials of `tokens` tokens, whatever the context.
size_t grouped_part_bytes(const Device *dev, const GroupedShape &s, int f32, int tokens) {
    return part_bytes_for(s, (size_t)tokens * s.heads, auto_splits(dev, s, f32, tokens, 1 << 30));
}
int grouped_counters(const GroupedShape &s, int tokens) { return tokens * s.kv_heads * head_groups(s); }

int grouped_attention_run(const Device *dev, const GroupedArgs &a, cudaStream_t st, int *launches) {
    const GroupedShape &s = a.s;
    const int M = a.nseq * a.T;
    int rc;
    if (!a.f32 && a.nseq == 1 && a.host_slot >= 0 && a.T >= kGroupedPrefillMin && grouped_prefills(s)) {
        rc = rows_launch<__nv_bfloat16>(a, st);
        if (rc != IM_OK) return rc;
        *launches += 2;
        const int dv = prefill_dv(s);
        return dv == 64 ? prefill_launch<64>(a, st) : dv == 128 ? prefill_launch<128>(a, st) : prefill_launch<256>(a, st);
    }
    const bool tc = !a.f32 && decode_tc(s);
    if (!tc && s.vP > kGsThreads * kGsCols) return fail(IM_ERR_INVALID, "grouped attention is built for value sizes up to %d (got %d)", kGsThreads * kGsCols, s.vdim);
    GroupedPart p;
    p.splits = auto_splits(dev, s, a.f32, M, a.splits_ctx);
    const size_t rows = (size_t)M * s.heads;
    while (p.splits > 1 && part_bytes_for(s, rows, p.splits) > a.part_bytes) p.splits--;
    if (part_bytes_for(s, rows, p.splits) > a.part_bytes) return fail(IM_ERR_BOUNDS, "grouped attention scratch is too small for %d tokens", M);
    p.po = a.part;
    p.pm = p.po + rows * p.splits * s.vP;
    p.pl = p.pm + rows * p.splits;
    if (!tc || a.T > 1) {
        rc = a.f32 ? rows_launch<float>(a, st) : rows_launch<__nv_bfloat16>(a, st);
        if (rc != IM_OK) return rc;
        *launches += 1;
    }
    if (tc) {
        *launches += 1;
        return head_tiles(s) == 2 ? decode_any<2>(a, p, st) : decode_any<1>(a, p, st);
    }
    *launches += 2;
    return a.f32 ? simt_launch<float>(a, p, st) : simt_launch<__nv_bfloat16>(a, p, st);
}

}  // namespace im
