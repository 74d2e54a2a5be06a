// Dense projections (bf16 with f32 accumulation, or true f32) with fused prologues and epilogues.
//   up to 15 tokens   dense_matvec_kernel: a warp (or several, K split) per pair of weight rows, 16-byte weight loads
//                     requested one step ahead, the activations staged once per CTA in shared memory; the staging can be
//                     the RMS norm of the f32 residual or the concatenation of two f32 vectors
//   16 tokens and more, bf16   dense_gemm_tc_kernel: tcgen05.mma, both operands by TMA into the 128-byte swizzle, f32
//                     accumulator in tensor memory, K split over the grid for few tokens
//   16 tokens and more, f32    dense_gemm_f32_kernel: register-tiled f32 FMA
// The epilogues (activation of some rows, gate * up pairs, residual add, bias, soft cap) work on the f32 sums.
#include <cuda.h>

#include <algorithm>

#include "stack.cuh"
#include "v2_device.cuh"

namespace im {

namespace {

// Two neighbouring rows n, n + 1 (n even) of token m.
template <typename T>
__device__ __forceinline__ void epi_pair(const DenseEpi &e, int m, int n, float v0, float v1, int N) {
    if (e.kind == kEpiProj) {
        if (n >= e.pair0) {
            static_cast<T *>(e.act)[(size_t)m * e.ldact + ((n - e.pair0) >> 1)] = from_f<T>((e.pair_silu ? silu_f(v0) : gelu_tanh_f(v0)) * v1);
        } else if (n >= e.f0) {
            float *f = e.xf + (size_t)m * e.ldx + (n - e.f0);
            f[0] = v0;
            if (n + 1 < N) f[1] = v1;
        } else {
            T *y = static_cast<T *>(e.y) + (size_t)m * e.ldy + n;
            if (n < e.silu_end) {
                v0 = silu_f(v0);
                v1 = silu_f(v1);
            }
            y[0] = from_f<T>(v0);
            if (n + 1 < N) y[1] = from_f<T>(v1);
        }
        return;
    }
    float *x = e.xf + (size_t)m * e.ldx + n;
    if (e.kind == kEpiResidual) {
        x[0] += v0;
        if (n + 1 < N) x[1] += v1;
        return;
    }
    if (e.bias) {
        v0 += e.bias[n];
        if (n + 1 < N) v1 += e.bias[n + 1];
    }
    if (e.cap > 0.0f) {
        v0 = e.cap * tanhf(v0 / e.cap);
        v1 = e.cap * tanhf(v1 / e.cap);
    }
    x[0] = v0;
    if (n + 1 < N) x[1] = v1;
}

// One row of the source as elements of type T (dst: K of them, then zeros up to ld), by the whole block.  keep: this block
// writes the row's new residual (kSrcAddNorm).
template <typename T>
__device__ __forceinline__ void stage_row(const DenseSrc &s, int m, int K, int ld, T *dst, float *sh, bool keep) {
    const int tid = threadIdx.x, nt = blockDim.x;
    if (s.kind == kSrcPlain) {
        constexpr int V = Vec16<T>::n;
        const T *x = static_cast<const T *>(s.x) + (size_t)m * s.ldx;
        const int kv = K / V;
        for (int i = tid; i < kv; i += nt) reinterpret_cast<uint4 *>(dst)[i] = reinterpret_cast<const uint4 *>(x)[i];
        for (int i = kv * V + tid; i < ld; i += nt) dst[i] = i < K ? x[i] : from_f<T>(0.0f);
        return;
    }
    const float *x = s.xf + (size_t)m * s.ldx;
    if (s.kind == kSrcConcat) {
        const float *x2 = s.xf2 + (size_t)m * s.ldx;
        for (int i = tid; i < ld; i += nt) dst[i] = from_f<T>(i < s.width ? x[i] : i < K ? x2[i - s.width] : 0.0f);
        return;
    }
    float ss = 0.0f;
    if (s.kind == kSrcAddNorm) {
        const float *add = s.xf2 ? s.xf2 + (size_t)m * s.ldx : nullptr;
        float inv = 0.0f;
        if (add) {
            for (int i = tid; i < K; i += nt) ss = fmaf(add[i], add[i], ss);
            inv = 1.0f / sqrtf(block_sum_f(ss, sh) / (float)K + s.eps);
        }
        auto sum = [&](int i) { return add ? x[i] + add[i] * inv * s.gamma[i] : x[i]; };
        float inv2 = 1.0f;
        if (s.gamma2) {
            ss = 0.0f;
            for (int i = tid; i < K; i += nt) {
                const float r = sum(i);
                ss = fmaf(r, r, ss);
            }
            inv2 = 1.0f / sqrtf(block_sum_f(ss, sh) / (float)K + s.eps);
        }
        float *out = keep && s.xout ? s.xout + (size_t)m * s.ldx : nullptr;
        for (int i = tid; i < ld; i += nt) {
            float r = 0.0f;
            if (i < K) {
                r = sum(i);
                if (out) out[i] = r;
                if (s.gamma2) r *= inv2 * s.gamma2[i];
            }
            dst[i] = from_f<T>(r);
        }
        return;
    }
    for (int i = tid; i < K; i += nt) ss = fmaf(x[i], x[i], ss);
    const float inv = 1.0f / sqrtf(block_sum_f(ss, sh) / (float)K + s.eps);
    for (int i = tid; i < ld; i += nt) dst[i] = from_f<T>(i < K ? x[i] * inv * s.gamma[i] : 0.0f);
}

constexpr int kMvThreads = 256, kMvWarps = kMvThreads / 32, kMvU = 4;

template <typename T, int NB>
__global__ void __launch_bounds__(kMvThreads, NB <= 4 ? 2 : 1) dense_matvec_kernel(const DenseWeight w, const DenseSrc src, const DenseEpi epi, int m0, int B, int KS) {
    extern __shared__ __align__(16) unsigned char dense_smem[];
    __shared__ float sh[32];
    __shared__ float red[kMvWarps][2][NB];
    constexpr int V = Vec16<T>::n;
    T *xs = reinterpret_cast<T *>(dense_smem);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int groups = kMvWarps / KS, grp = warp / KS, ks = warp % KS;
    const int kv = w.ld / V, nit = (kv + 32 * kMvU * KS - 1) / (32 * kMvU * KS);
    const int ntiles = (w.N + 2 * groups - 1) / (2 * groups);
    const T *W = static_cast<const T *>(w.w);
    uint4 nxt[2][kMvU] = {};
    // Every address is clamped into the matrix (rows past the end repeat the last one, columns past the end the last
    // vector): the streaming load is inline assembly without side effects, which a compiler may move above a guard.
    auto load = [&](int tile, int it) {
        if (tile >= ntiles) return;
        const int n0 = (tile * groups + grp) * 2;
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const T *row = W + (size_t)min(n0 + r, w.N - 1) * w.ld;
#pragma unroll
            for (int u = 0; u < kMvU; u++) nxt[r][u] = ldg_stream_v4(row + (size_t)min(((it * KS + ks) * kMvU + u) * 32 + lane, kv - 1) * V);
        }
    };
    pdl_trigger();
    load(blockIdx.x, 0);  // weights are constants: requested before the predecessor has finished
    pdl_wait();
    for (int b = 0; b < B; b++) stage_row<T>(src, m0 + b, w.K, w.ld, xs + (size_t)b * w.ld, sh, blockIdx.x == 0);
    __syncthreads();
    for (int tile = blockIdx.x; tile < ntiles; tile += gridDim.x) {
        const int n0 = (tile * groups + grp) * 2;
        float acc[2][NB];
#pragma unroll
        for (int b = 0; b < NB; b++) acc[0][b] = acc[1][b] = 0.0f;
        for (int it = 0; it < nit; it++) {
            uint4 cur[2][kMvU];
#pragma unroll
            for (int r = 0; r < 2; r++)
#pragma unroll
                for (int u = 0; u < kMvU; u++) cur[r][u] = nxt[r][u];
            if (it + 1 < nit) load(tile, it + 1);
            else load(tile + (int)gridDim.x, 0);
#pragma unroll
            for (int u = 0; u < kMvU; u++) {
                const int i = ((it * KS + ks) * kMvU + u) * 32 + lane;
                if (i < kv) {
                    float w0[V], w1[V];
                    Vec16<T>::unpack(cur[0][u], w0);
                    Vec16<T>::unpack(cur[1][u], w1);
#pragma unroll
                    for (int b = 0; b < NB; b++) {
                        if (b < B) {
                            float xv[V];
                            Vec16<T>::unpack(*reinterpret_cast<const uint4 *>(xs + (size_t)b * w.ld + (size_t)i * V), xv);
#pragma unroll
                            for (int j = 0; j < V; j++) {
                                acc[0][b] = fmaf(w0[j], xv[j], acc[0][b]);
                                acc[1][b] = fmaf(w1[j], xv[j], acc[1][b]);
                            }
                        }
                    }
                }
            }
        }
#pragma unroll
        for (int b = 0; b < NB; b++) {
            acc[0][b] = warp_sum(acc[0][b]);
            acc[1][b] = warp_sum(acc[1][b]);
        }
        if (KS > 1) {
            if (lane == 0)
#pragma unroll
                for (int b = 0; b < NB; b++) {
                    red[warp][0][b] = acc[0][b];
                    red[warp][1][b] = acc[1][b];
                }
            __syncthreads();
            if (ks == 0)
#pragma unroll
                for (int b = 0; b < NB; b++)
                    for (int k = 1; k < KS; k++) {
                        acc[0][b] += red[warp + k][0][b];
                        acc[1][b] += red[warp + k][1][b];
                    }
            __syncthreads();
        }
        if (ks == 0 && n0 < w.N)
#pragma unroll
            for (int b = 0; b < NB; b++)
                if (b < B && lane == b) epi_pair<T>(epi, m0 + b, n0, acc[0][b], acc[1][b], w.N);
    }
}

// The source as a matrix of elements (tokens that a GEMM reads): one CTA per token.
template <typename T>
__global__ void __launch_bounds__(256) dense_stage_kernel(const DenseSrc src, int K, int ld, T *__restrict__ out) {
    __shared__ float sh[32];
    pdl_trigger();
    pdl_wait();
    stage_row<T>(src, blockIdx.x, K, ld, out + (size_t)blockIdx.x * ld, sh, true);
}

// ---- tcgen05 GEMM ----------------------------------------------------------------------------------------------------
// Persistent: a CTA walks work items (weight tile, token tile, K slice), token tiles of one weight tile next to each other
// so that the weights stream from memory once.  Two accumulators in tensor memory: the epilogue warps convert and store one
// item while the next one's products run.
constexpr int kDM = 128, kDK = 64;  // weight rows and columns of a stage (one 128-byte swizzle row)
constexpr int kDEpi = 8;            // epilogue warps: warp w reads tensor-memory lanes 32 (w % 4) .., half w / 4 of the tokens
constexpr int kDThreads = (kDEpi + 2) * 32;  // ... then one warp for the copies, one for tensor memory + MMA issue
template <int TN>
constexpr int dense_stages() { return TN >= 256 ? 4 : TN == 128 ? 3 : 4; }
template <int TN>
constexpr int dense_gemm_smem() { return 1024 + dense_stages<TN>() * (kDM * 128 + TN * 128) + (2 * dense_stages<TN>() + 4) * 8 + 16; }
template <int TN>
constexpr int dense_ctas_per_sm() { return TN >= 256 ? 1 : 2; }

__device__ __forceinline__ uint64_t dense_desc_sw128(uint32_t smem_addr) {
    // K-major, 128-byte swizzle: start >> 4, leading offset 1, stride offset 1024 B >> 4, version 1, layout 2 (see gemm_tc.cu)
    return (uint64_t)((smem_addr & 0x3FFFFu) >> 4) | (1ull << 16) | (64ull << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void dense_mma(uint32_t tmem_d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t accumulate) {
    asm volatile("{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
                 "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5}, p;\n\t}\n" ::"r"(tmem_d), "l"(a), "l"(b), "r"(idesc),
                 "r"(accumulate), "r"(0)
                 : "memory");
}
__device__ __forceinline__ void dense_commit(uint64_t *bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void dense_tmem_ld16(uint32_t taddr, float (&v)[16]) {
    uint32_t r[16];
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32"
        "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];\n"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
          "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
        : "r"(taddr));
    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
    for (int i = 0; i < 16; i++) v[i] = __uint_as_float(r[i]);
}
__device__ __forceinline__ void dense_tma_2d(void *dst, const CUtensorMap *map, int x, int y, uint64_t *bar) {
    // x is a multiple of 64 elements (128 bytes)
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(smem_u32(dst)), "l"(map),
                 "r"(x), "r"(y), "r"(smem_u32(bar))
                 : "memory");
}
// bf16 epilogues: z sigmoid(z), and gelu_tanh(z) = z / (1 + exp(-2 u)), u = sqrt(2 / pi) (z + 0.044715 z^3); the error of the
// fast exponential and quotient (about 1e-6) is far below the bf16 result's rounding
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
__device__ __forceinline__ float pair_act_fast(float z, float up, bool silu) {
    if (silu) return silu_fast(z) * up;
    const float w = -1.5957691216057308f * z * fmaf(0.044715f * z, z, 1.0f);
    return __fdividef(z * up, 1.0f + __expf(fminf(w, 80.0f)));
}

struct DenseGemm {
    int N, M, kblocks, kb_per;  // kblocks: 64-column blocks of K; kb_per: of one K slice
    int mtiles, ntiles, slices;
    float *partial;             // [slices][M][N] when K is split
    int *err;
    DenseEpi epi;
};

// 16 tokens m .. m + 15 of row n (one per lane) of the f32 sums
__device__ __forceinline__ void dense_store16(const DenseGemm &p, int z, int n, int n_warp, int m, const float (&v)[16]) {
    typedef __nv_bfloat16 T;
    const DenseEpi &e = p.epi;
    const int lane = threadIdx.x & 31, left = p.M - m;
    if (p.partial) {
        if (n < p.N) {
            float *dst = p.partial + ((size_t)z * p.M + m) * p.N + n;
#pragma unroll
            for (int i = 0; i < 16; i++)
                if (i < left) dst[(size_t)i * p.N] = v[i];
        }
    } else if (e.kind == kEpiProj) {
        if (n_warp + 31 >= e.pair0) {
            // (gate, up) sit in neighbouring lanes: of two tokens, the even lane takes the first, the odd lane the second
            // (pair0 is a multiple of eight: no pair straddles it)
            T *act = static_cast<T *>(e.act) + (size_t)m * e.ldact + ((n - e.pair0) >> 1);
            T *y = static_cast<T *>(e.y) + (size_t)m * e.ldy + n;
            const bool odd = lane & 1, pair = n >= e.pair0;
#pragma unroll
            for (int i = 0; i < 16; i += 2) {
                const float got = __shfl_xor_sync(0xffffffffu, odd ? v[i] : v[i + 1], 1);
                if (pair) {
                    const float r = odd ? pair_act_fast(got, v[i + 1], e.pair_silu) : pair_act_fast(v[i], got, e.pair_silu);
                    if (n < p.N && i + odd < left) act[(size_t)(i + odd) * e.ldact] = from_f<T>(r);
                } else {
#pragma unroll
                    for (int j = 0; j < 2; j++)
                        if (i + j < left) {
                            if (n >= e.f0) e.xf[(size_t)(m + i + j) * e.ldx + (n - e.f0)] = v[i + j];
                            else y[(size_t)(i + j) * e.ldy] = from_f<T>(n < e.silu_end ? silu_fast(v[i + j]) : v[i + j]);
                        }
                }
            }
        } else {
            T *y = static_cast<T *>(e.y) + (size_t)m * e.ldy + n;
            const bool act = n < e.silu_end;
            if (n < p.N && n >= e.f0) {
                float *f = e.xf + (size_t)m * e.ldx + (n - e.f0);
#pragma unroll
                for (int i = 0; i < 16; i++)
                    if (i < left) f[(size_t)i * e.ldx] = v[i];
            } else if (n < p.N) {
#pragma unroll
                for (int i = 0; i < 16; i++)
                    if (i < left) y[(size_t)i * e.ldy] = from_f<T>(act ? silu_fast(v[i]) : v[i]);
            }
        }
    } else if (n < p.N) {
        float *x = e.xf + (size_t)m * e.ldx + n;
        if (e.kind == kEpiResidual) {
            float old[16];
#pragma unroll
            for (int i = 0; i < 16; i++) old[i] = i < left ? x[(size_t)i * e.ldx] : 0.0f;
#pragma unroll
            for (int i = 0; i < 16; i++)
                if (i < left) x[(size_t)i * e.ldx] = old[i] + v[i];
        } else {
            const float b = e.bias ? e.bias[n] : 0.0f;
#pragma unroll
            for (int i = 0; i < 16; i++) {
                float r = v[i] + b;
                if (e.cap > 0.0f) r = e.cap * tanhf(r / e.cap);
                if (i < left) x[(size_t)i * e.ldx] = r;
            }
        }
    }
}

// D[128 weight rows x TN tokens] += W[128 x 64] X[TN x 64]^T per stage.
template <int TN>
__global__ void __launch_bounds__(kDThreads, dense_ctas_per_sm<TN>()) dense_gemm_tc_kernel(const DenseGemm p, const __grid_constant__ CUtensorMap ta,
                                                                                         const __grid_constant__ CUtensorMap tb) {
    constexpr int S = dense_stages<TN>();
    constexpr int kA = kDM * 128, kB = TN * 128, kCols = 2 * TN;
    extern __shared__ __align__(1024) unsigned char dense_gemm_raw[];
    unsigned char *smem = reinterpret_cast<unsigned char *>((reinterpret_cast<uintptr_t>(dense_gemm_raw) + 1023) & ~(uintptr_t)1023);
    unsigned char *As = smem, *Bs = smem + S * kA;
    uint64_t *full = reinterpret_cast<uint64_t *>(Bs + S * kB), *empty = full + S, *tfull = empty + S, *tempty = tfull + 2;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(tempty + 2);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    pdl_trigger();
    if (tid == 0) {
        for (int i = 0; i < S; i++) {
            mbar_init(&full[i], 1);
            mbar_init(&empty[i], 1);
        }
        for (int i = 0; i < 2; i++) {
            mbar_init(&tfull[i], 1);
            mbar_init(&tempty[i], kDEpi);
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == kDEpi + 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(kCols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem_d = *tmem_slot;
    pdl_wait();
    const int items = p.mtiles * p.ntiles * p.slices;
    bool ok = true;
    if (warp == kDEpi) {
        int it = 0;
        for (int w = blockIdx.x; w < items; w += gridDim.x) {
            const int m0 = w % p.mtiles * TN, n0 = w / p.mtiles % p.ntiles * kDM, kb0 = w / (p.mtiles * p.ntiles) * p.kb_per;
            const int kb1 = min(p.kblocks, kb0 + p.kb_per);
            for (int kb = kb0; kb < kb1; kb++, it++) {
                const int s = it % S, use = it / S;
                if (ok && use > 0 && !mbar_wait_warp(&empty[s], (use - 1) & 1, p.err)) ok = false;
                if (lane == 0 && ok) {
                    mbar_expect_tx(&full[s], (uint32_t)(kA + kB));
                    dense_tma_2d(As + (size_t)s * kA, &ta, kb * kDK, n0, &full[s]);
                    dense_tma_2d(Bs + (size_t)s * kB, &tb, kb * kDK, m0, &full[s]);
                }
                __syncwarp();
            }
        }
    } else if (warp == kDEpi + 1) {
        // f32 accumulator, bf16 operands, both K-major, N >> 3 in bits 17-22, M >> 4 in bits 24-28
        constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(TN >> 3) << 17) | ((uint32_t)(kDM >> 4) << 24);
        int it = 0, cnt = 0;
        for (int w = blockIdx.x; w < items; w += gridDim.x, cnt++) {
            const int kb0 = w / (p.mtiles * p.ntiles) * p.kb_per, kb1 = min(p.kblocks, kb0 + p.kb_per);
            const int acc = cnt & 1, use = cnt >> 1;
            if (ok && use > 0 && !mbar_wait_warp(&tempty[acc], (use - 1) & 1, p.err)) ok = false;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            for (int kb = kb0; kb < kb1; kb++, it++) {
                const int s = it % S;
                if (ok && !mbar_wait_warp(&full[s], (it / S) & 1, p.err)) ok = false;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                if (lane == 0 && ok) {
                    const uint32_t a0 = smem_u32(As + (size_t)s * kA), b0 = smem_u32(Bs + (size_t)s * kB);
#pragma unroll
                    for (int j = 0; j < 4; j++)
                        dense_mma(tmem_d + (uint32_t)(acc * TN), dense_desc_sw128(a0 + j * 32), dense_desc_sw128(b0 + j * 32), idesc, (kb > kb0 || j > 0) ? 1u : 0u);
                    dense_commit(&empty[s]);
                    if (kb == kb1 - 1) dense_commit(&tfull[acc]);
                }
                __syncwarp();
            }
        }
    } else {
        int cnt = 0;
        for (int w = blockIdx.x; w < items; w += gridDim.x, cnt++) {
            const int m0 = w % p.mtiles * TN, n_warp = w / p.mtiles % p.ntiles * kDM + (warp & 3) * 32, z = w / (p.mtiles * p.ntiles);
            const int acc = cnt & 1;
            if (ok && !mbar_wait_warp(&tfull[acc], (cnt >> 1) & 1, p.err)) ok = false;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            if (ok) {
                const int c_begin = (warp >> 2) * (TN / 2);
#pragma unroll 1
                for (int c = c_begin; c < c_begin + TN / 2 && m0 + c < p.M; c += 16) {
                    float v[16];
                    dense_tmem_ld16(tmem_d + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)(acc * TN + c), v);
                    dense_store16(p, z, n_warp + lane, n_warp, m0 + c, v);
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(&tempty[acc]);
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == kDEpi + 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_d), "r"(kCols) : "memory");
    }
}

// K slices added in order, then the epilogue; one thread per (token, pair of rows)
template <typename T>
__global__ void __launch_bounds__(256) dense_splitk_reduce_kernel(const float *__restrict__ partial, const DenseEpi epi, int M, int N, int slices) {
    pdl_trigger();
    pdl_wait();
    const int half = (N + 1) / 2;
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)M * half) return;
    const int m = (int)(i / half), n = 2 * (int)(i % half);
    float v0 = 0.0f, v1 = 0.0f;
    for (int z = 0; z < slices; z++) {
        const float *q = partial + ((size_t)z * M + m) * N + n;
        v0 += q[0];
        if (n + 1 < N) v1 += q[1];
    }
    epi_pair<T>(epi, m, n, v0, v1, N);
}

// ---- f32 GEMM: 64 tokens x 64 rows per CTA, 4 x 4 per thread -----------------------------------------------------------
__global__ void __launch_bounds__(256) dense_gemm_f32_kernel(const DenseWeight w, const float *__restrict__ x, int ldx, const DenseEpi epi, int M) {
    __shared__ __align__(16) float xs[16][68], ws[16][68];
    pdl_trigger();
    pdl_wait();
    const float *W = static_cast<const float *>(w.w);
    const int n0 = blockIdx.x * 64, m0 = blockIdx.y * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < w.K; k0 += 16) {
        for (int i = threadIdx.x; i < 1024; i += 256) {
            const int r = i >> 4, k = i & 15;
            xs[k][r] = (m0 + r < M && k0 + k < w.K) ? x[(size_t)(m0 + r) * ldx + k0 + k] : 0.0f;
            ws[k][r] = (n0 + r < w.N && k0 + k < w.K) ? W[(size_t)(n0 + r) * w.ld + k0 + k] : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; k++) {
            const float4 a = *reinterpret_cast<const float4 *>(&xs[k][4 * ty]), b = *reinterpret_cast<const float4 *>(&ws[k][4 * tx]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
        __syncthreads();
    }
    for (int i = 0; i < 4; i++) {
        const int m = m0 + 4 * ty + i;
        if (m >= M) break;
        for (int j = 0; j < 4; j += 2) {
            const int n = n0 + 4 * tx + j;
            if (n < w.N) epi_pair<float>(epi, m, n, acc[i][j], acc[i][j + 1], w.N);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(256) stack_embed_kernel(const uint32_t *__restrict__ tokens, const T *__restrict__ table, int ld, const float *__restrict__ gamma,
                                                          float scale, float *__restrict__ x, float *__restrict__ x0, int W, uint32_t vocab, float eps) {
    __shared__ float sh[32];
    pdl_trigger();
    pdl_wait();
    const uint32_t tok = tokens[blockIdx.x];
    const T *row = table + (size_t)(tok < vocab ? tok : 0) * ld;
    const bool live = tok < vocab;
    float ss = 0.0f, inv = scale;
    if (gamma) {
        for (int i = threadIdx.x; i < W; i += blockDim.x) {
            const float v = live ? to_f<T>(row[i]) : 0.0f;
            ss = fmaf(v, v, ss);
        }
        inv = 1.0f / sqrtf(block_sum_f(ss, sh) / (float)W + eps);
    }
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
        float v = (live ? to_f<T>(row[i]) : 0.0f) * inv;
        if (gamma) v *= gamma[i];
        x[(size_t)blockIdx.x * W + i] = v;
        x0[(size_t)blockIdx.x * W + i] = v;
    }
}

// ---- host ------------------------------------------------------------------------------------------------------------
typedef CUresult (*TmapEncodeFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *, const cuuint32_t *,
                                 const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
TmapEncodeFn tmap_encode() {
    static TmapEncodeFn fn = [] {
        void *f = nullptr;
        cudaDriverEntryPointQueryResult q = cudaDriverEntryPointSymbolNotFound;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &f, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) f = nullptr;
        return reinterpret_cast<TmapEncodeFn>(f);
    }();
    return fn;
}
// bf16 [rows, cols] with row stride ld (a multiple of 8): boxes of 64 columns x box_rows, zeros outside
int bf16_tmap(const void *base, int rows, int cols, int ld, int box_rows, CUtensorMap *out) {
    TmapEncodeFn enc = tmap_encode();
    if (!enc) return fail(IM_ERR_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
    const cuuint64_t gdim[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    const cuuint64_t gstride[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {64u, (cuuint32_t)box_rows}, es[2] = {1u, 1u};
    const CUresult r = enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), gdim, gstride, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                           CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail(IM_ERR_CUDA, "cuTensorMapEncodeTiled failed (%d) for bf16 [%d, %d] stride %d", (int)r, rows, cols, ld);
    return IM_OK;
}

template <int TN>
int gemm_launch(const Device *dev, DenseGemm p, const DenseWeight &w, const void *x, int ldx, int slices, cudaStream_t st) {
    alignas(64) CUtensorMap ta, tb;
    int rc = bf16_tmap(w.w, w.N, w.K, w.ld, kDM, &ta);
    if (rc != IM_OK) return rc;
    rc = bf16_tmap(x, p.M, w.K, ldx, TN, &tb);
    if (rc != IM_OK) return rc;
    p.mtiles = (p.M + TN - 1) / TN;
    p.ntiles = (p.N + kDM - 1) / kDM;
    p.slices = slices;
    const int ctas = std::min(p.mtiles * p.ntiles * slices, dev->sm_count * dense_ctas_per_sm<TN>());
    IM_CUDA_CHECK(launch_k(dense_gemm_tc_kernel<TN>, dim3(ctas), dim3(kDThreads), (size_t)dense_gemm_smem<TN>(), st, p, ta, tb));
    if (p.partial) {
        const size_t n = (size_t)p.M * ((p.N + 1) / 2);
        IM_CUDA_CHECK(launch_k(dense_splitk_reduce_kernel<__nv_bfloat16>, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, st, (const float *)p.partial, p.epi, p.M, p.N,
                               slices));
    }
    return IM_OK;
}

template <typename T, int NB>
int matvec_launch(const Device *dev, const DenseWeight &w, const DenseSrc &src, const DenseEpi &epi, int m0, int B, cudaStream_t st) {
    const size_t smem = (size_t)NB * w.ld * sizeof(T);
    const int pairs = (w.N + 1) / 2, ctas = dev->sm_count * (NB <= 4 && smem <= 100 * 1024 ? 2 : 1);
    int KS = 1;
    while (KS < kMvWarps && pairs * KS < ctas * kMvWarps) KS *= 2;
    const int groups = kMvWarps / KS, ntiles = (w.N + 2 * groups - 1) / (2 * groups);
    IM_CUDA_CHECK(launch_k(dense_matvec_kernel<T, NB>, dim3(std::min(ntiles, ctas)), dim3(kMvThreads), smem, st, w, src, epi, m0, B, KS));
    return IM_OK;
}
constexpr size_t kMvSmemMax = 200 * 1024;

template <typename T>
int matvec_any(const Device *dev, const DenseWeight &w, const DenseSrc &src, const DenseEpi &epi, int M, cudaStream_t st) {
    int cap = kDenseMaxRows;
    while (cap > 1 && (size_t)cap * w.ld * sizeof(T) > kMvSmemMax) cap /= 2;
    if ((size_t)w.ld * sizeof(T) > kMvSmemMax) return fail(IM_ERR_INVALID, "a projection with %d input columns does not fit shared memory", w.K);
    for (int m0 = 0; m0 < M;) {
        const int B = std::min(M - m0, cap);
        int rc;
        if (B > 4) rc = matvec_launch<T, 8>(dev, w, src, epi, m0, B, st);
        else if (B > 2) rc = matvec_launch<T, 4>(dev, w, src, epi, m0, B, st);
        else if (B > 1) rc = matvec_launch<T, 2>(dev, w, src, epi, m0, B, st);
        else rc = matvec_launch<T, 1>(dev, w, src, epi, m0, B, st);
        if (rc != IM_OK) return rc;
        m0 += B;
    }
    return IM_OK;
}

}  // namespace

int dense_prepare(const Device *dev) {
    static DeviceOnce once;
    if (!once.first(dev->ordinal)) return IM_OK;
    const int mv = (int)kMvSmemMax;
#define IM_SMEM(k, b) IM_CUDA_CHECK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, b))
    IM_SMEM((dense_matvec_kernel<__nv_bfloat16, 1>), mv); IM_SMEM((dense_matvec_kernel<__nv_bfloat16, 2>), mv);
    IM_SMEM((dense_matvec_kernel<__nv_bfloat16, 4>), mv); IM_SMEM((dense_matvec_kernel<__nv_bfloat16, 8>), mv);
    IM_SMEM((dense_matvec_kernel<float, 1>), mv); IM_SMEM((dense_matvec_kernel<float, 2>), mv);
    IM_SMEM((dense_matvec_kernel<float, 4>), mv); IM_SMEM((dense_matvec_kernel<float, 8>), mv);
    IM_SMEM(dense_gemm_tc_kernel<256>, dense_gemm_smem<256>()); IM_SMEM(dense_gemm_tc_kernel<128>, dense_gemm_smem<128>());
    IM_SMEM(dense_gemm_tc_kernel<64>, dense_gemm_smem<64>()); IM_SMEM(dense_gemm_tc_kernel<32>, dense_gemm_smem<32>());
#undef IM_SMEM
    return IM_OK;
}

int dense_launches(int M, int K, int src_kind) {
    (void)K;
    return M >= kDenseGemmMin ? 1 + (src_kind != kSrcPlain) : (M + kDenseMaxRows - 1) / kDenseMaxRows;
}

int dense_project(const Device *dev, const DenseWeight &w, const DenseSrc &src, const DenseEpi &epi, int M, void *h_scratch, cudaStream_t st) {
    if (M <= 0) return IM_OK;
    const int ldv = 16 / (int)elem_size(w.f32);
    if (src.kind == kSrcPlain && src.ldx % ldv != 0) return fail(IM_ERR_INVALID, "activation rows must be 16-byte aligned");
    if (M < kDenseGemmMin) return w.f32 ? matvec_any<float>(dev, w, src, epi, M, st) : matvec_any<__nv_bfloat16>(dev, w, src, epi, M, st);
    const void *x = src.x;
    int ldx = src.ldx;
    if (src.kind != kSrcPlain) {
        if (w.f32) IM_CUDA_CHECK(launch_k(dense_stage_kernel<float>, dim3(M), dim3(256), 0, st, src, w.K, w.ld, static_cast<float *>(h_scratch)));
        else IM_CUDA_CHECK(launch_k(dense_stage_kernel<__nv_bfloat16>, dim3(M), dim3(256), 0, st, src, w.K, w.ld, static_cast<__nv_bfloat16 *>(h_scratch)));
        x = h_scratch;
        ldx = w.ld;
    }
    if (w.f32) {
        IM_CUDA_CHECK(launch_k(dense_gemm_f32_kernel, dim3((w.N + 63) / 64, (M + 63) / 64), dim3(256), 0, st, w, static_cast<const float *>(x), ldx, epi, M));
        return IM_OK;
    }
    DenseGemm p{};
    p.N = w.N; p.M = M; p.kblocks = (w.K + kDK - 1) / kDK; p.kb_per = p.kblocks; p.err = dev->err_flag; p.epi = epi;
    const int tiles = (w.N + kDM - 1) / kDM;
    int slices = 1;
    if (M <= 128) {  // few tokens: split K until the grid covers the GPU, at least four blocks a slice
        const int mt = M <= 32 ? 1 : M <= 64 ? 1 : (M + 127) / 128;
        slices = std::max(1, std::min(dev->sm_count / (tiles * mt), p.kblocks / 4));
        while (slices > 1 && (size_t)slices * M * w.N * sizeof(float) > kGemmPartialBytes) slices--;
        if (slices > 1) {
            p.kb_per = (p.kblocks + slices - 1) / slices;
            slices = (p.kblocks + p.kb_per - 1) / p.kb_per;
            p.partial = dev->gemm_partial;
        }
    }
    const long long ctas256 = (long long)tiles * ((M + 255) / 256);
    if (M > 128 && ctas256 >= dev->sm_count) return gemm_launch<256>(dev, p, w, x, ldx, slices, st);
    if (M > 64) return gemm_launch<128>(dev, p, w, x, ldx, slices, st);
    if (M > 32) return gemm_launch<64>(dev, p, w, x, ldx, slices, st);
    return gemm_launch<32>(dev, p, w, x, ldx, slices, st);
}

int stack_embed(const uint32_t *tokens, const void *table, int f32, int ld, const float *gamma, float scale, float *x, float *x0, int width, uint32_t vocab, float eps,
                int M, cudaStream_t st) {
    if (M <= 0) return IM_OK;
    if (f32)
        IM_CUDA_CHECK(launch_k(stack_embed_kernel<float>, dim3(M), dim3(256), 0, st, tokens, static_cast<const float *>(table), ld, gamma, scale, x, x0, width, vocab, eps));
    else
        IM_CUDA_CHECK(launch_k(stack_embed_kernel<__nv_bfloat16>, dim3(M), dim3(256), 0, st, tokens, static_cast<const __nv_bfloat16 *>(table), ld, gamma, scale, x, x0,
                               width, vocab, eps));
    return IM_OK;
}

}  // namespace im
