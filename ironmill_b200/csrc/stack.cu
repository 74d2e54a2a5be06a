// Models given as a list of layers (im_cuda_model_create_stack): the Gizizen and Luvatar designs and relatives.
//   x = rms(embed[token]) g (or embed[token] * scale), x0 = x
//   looped passes begin with  x <- W_in [x; x0] + step[pass]
//   every layer, parallel     x <- x + mixer(n) + ffn(n),  n = rms(x) g
//            or post-norm     x <- x + rms(mixer(x)) g1,  x <- x + rms(ffn(x)) g2
//   logits = cap tanh(head rms(x) g / cap)
// The residual is f32.  A parallel layer is a handful of launches:
//   1  norm + every projection that reads n, in one: [mixer rows | (gate, up) pairs], the feed-forward's activation in the
//      epilogue
//   2  the mixer proper (latent_attn.cu, linear_attn.cu, grouped_attn.cu), its heads landing beside the feed-forward's activations
//   3  [W_o | W_down] on that row, added to the residual
// A post-norm layer leaves every sublayer's output in a buffer of its own; whoever reads the residual next norms and adds it on
// the way in (the prologue of the next projection, which also writes the new residual):
//   1  mixer rows   2  the mixer   3  W_o   4  (gate, up) pairs   5  W_down
// Slots, captured decode steps, greedy decoding and the entry points of a step are the session's (session.cu).
#include <math.h>
#include <string.h>

#include <algorithm>
#include <array>
#include <map>
#include <new>
#include <set>
#include <string>
#include <vector>

#include "session.cuh"
#include "stack.cuh"

namespace im {

namespace {

constexpr int kStackChunk = 2048;     // most tokens of one forward pass
constexpr int kStackChunkWide = 256;  // ... where every token keeps absorbed queries and partial sums in scratch
constexpr size_t kExpandBytes = (size_t)256 << 20;  // expanded keys and values of a prompt chunk (at least one head)

struct StackLayer {
    im_stack_layer c{};
    std::vector<double> decay;
    LatentShape ls{};
    LinearShape ns{};
    GroupedShape gs{};
    int pair0 = 0, mixP = 0, ffP = 0;  // mixer rows of the input projection; columns of the output projection
    int silu_end = 0, f0 = 1 << 30;    // rows that go through SiLU; first row that goes out as f32
    DenseWeight w_in, w_out;           // parallel: [mixer | feed-forward] both
    DenseWeight w_gu, w_down;          // post-norm
    void *ukv = nullptr;
    float *norm1 = nullptr, *norm2 = nullptr, *c_norm = nullptr, *sink = nullptr, *o_norm = nullptr, *pows = nullptr;
    float *q_norm = nullptr, *k_norm = nullptr, *a2 = nullptr, *a2b = nullptr;
    const float *cosc = nullptr, *sinc = nullptr;
    bool linear() const { return c.mixer == IM_MIXER_LINEAR || c.mixer == IM_MIXER_GATED; }
    int value_pad() const { return c.mixer == IM_MIXER_LATENT ? ls.vP : c.mixer == IM_MIXER_GROUPED ? gs.vP : ns.vP; }
};
struct StackRun {  // one pass through a layer: its place in the order, its cache or state
    int layer = 0, pass = -1;
    bool opens = false;  // first layer of a looped pass
    void *cache = nullptr, *vcache = nullptr;  // grouped attention: keys, values (those of another run with kv_from)
};

__global__ void __launch_bounds__(256) rms_rows_kernel(const float *__restrict__ x, const float *__restrict__ g, float *__restrict__ out, int W, float eps) {
    __shared__ float sh[32];
    pdl_trigger();
    pdl_wait();
    const float *r = x + (size_t)blockIdx.x * W;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < W; i += blockDim.x) ss = fmaf(r[i], r[i], ss);
    const float inv = 1.0f / sqrtf(block_sum_f(ss, sh) / (float)W + eps);
    for (int i = threadIdx.x; i < W; i += blockDim.x) out[(size_t)blockIdx.x * W + i] = r[i] * inv * g[i];
}

}  // namespace

struct StackModel : im_model {
    im_stack_config sc{};
    std::vector<StackLayer> layers;
    std::vector<StackRun> runs;
    std::set<std::string> missing;
    int f32 = 0, W = 0;
    DenseWeight embed, head, loop_in;
    float *embed_norm = nullptr, *final_norm = nullptr, *loop_step = nullptr;
    float *x = nullptr, *x_alt = nullptr, *x0 = nullptr, *sub = nullptr, *a1 = nullptr, *decays = nullptr, *chunk_states = nullptr;
    unsigned *counters = nullptr;
    float *rec_o = nullptr, *seg_sums = nullptr, *part = nullptr, *logits = nullptr, *rows = nullptr, *hidden = nullptr;
    void *y = nullptr, *cat = nullptr, *h = nullptr, *qabs = nullptr, *kv = nullptr;
    int ldy = 0, ldcat = 0;
    int lda1 = 0;
    size_t part_bytes = 0, kv_bytes = 0, chunk_bytes = 0;
    bool has_state = false, post = false;  // post: post-norm blocks
    const float *last_x = nullptr;  // residual rows the last step's logits came from
    int last_rows = 0;
    std::map<std::array<double, 8>, std::pair<float *, float *>> rot_tables;

    int forward(int nseq, int T, cudaStream_t st, int *launches, Prof *prof, bool all_logits, const int *slots) override;
    int finalize() override;
    int alloc_logits_rows() override {
        IM_TRY(alloc((void **)&rows, (size_t)kAllLogitsChunk * cfg.vocab_size * 4));
        logits_rows = rows;
        return IM_OK;
    }
    bool recurrent() const override { return has_state; }
    int hidden_rows(int n, float *out_host) override;
    size_t step_bytes(int ctx, int batch) const override;
    const char *family() const override { return "stack"; }

    int dense_alloc(DenseWeight *w, int N, int K) {
        w->N = N; w->K = K; w->ld = round_up(K, 8); w->f32 = f32;
        const size_t n = (size_t)N * w->ld * elem_size(f32);
        IM_TRY(alloc(&w->w, n));
        IM_CUDA_CHECK(cudaMemset(w->w, 0, n));
        return IM_OK;
    }
    int load(const std::string &name, const void *data, int dtype, const std::vector<int64_t> &shape);
    int rot_table(const im_stack_layer &c, const float **cosc, const float **sinc);
    int mix(const StackRun &r, int nseq, int T, const int *slots, cudaStream_t st, int *nl);
    int logits_of(DenseSrc src, int row, int n, float *out, cudaStream_t st, int *nl);
};

namespace {

float bf16_value(uint16_t b) {
    const uint32_t u = (uint32_t)b << 16;
    float f;
    memcpy(&f, &u, 4);
    return f;
}
uint16_t bf16_bits(float f) {  // round to nearest, ties to even; NaN stays NaN
    uint32_t u;
    memcpy(&u, &f, 4);
    if ((u & 0x7fffffffu) > 0x7f800000u) return (uint16_t)((u >> 16) | 0x40u);
    return (uint16_t)((u + 0x7fffu + ((u >> 16) & 1u)) >> 16);
}
float source_value(const void *p, int dtype, size_t i) {
    if (dtype == IM_DTYPE_BF16) return bf16_value(static_cast<const uint16_t *>(p)[i]);
    if (dtype == IM_DTYPE_F16) return __half2float(static_cast<const __half *>(p)[i]);
    return static_cast<const float *>(p)[i];
}

// A tensor [rows, cols] on its way into a matrix whose rows and columns come in padded blocks: source row r goes to row
// (r / rb) * rbP + r % rb (times row_step), source column k to (k / cb) * cbP + k % cb, from (row0, col0) on.
struct Placement {
    int rb = 0, rbP = 0, cb = 0, cbP = 0;
    int row0 = 0, col0 = 0, row_step = 1;
};
int place(void *dst, int ld, int f32, const void *src, int dtype, int R, int C, Placement p) {
    if (!p.rb) p.rb = p.rbP = R;
    if (!p.cb) p.cb = p.cbP = C;
    const int nb = (C + p.cb - 1) / p.cb, width = nb * p.cbP;
    const size_t es = elem_size(f32);
    std::vector<unsigned char> buf;
    const bool raw = !f32 && dtype == IM_DTYPE_BF16;
    for (int r0 = 0; r0 < R; r0 += p.rb) {  // a block of rows is evenly spaced in the destination
        const int n = std::min(p.rb, R - r0);
        buf.assign((size_t)n * width * es, 0);
        for (int r = 0; r < n; r++)
            for (int c0 = 0; c0 < C; c0 += p.cb) {
                const int m = std::min(p.cb, C - c0);
                const size_t from = (size_t)(r0 + r) * C + c0, to = (size_t)r * width + (size_t)(c0 / p.cb) * p.cbP;
                if (raw) memcpy(buf.data() + to * 2, static_cast<const uint16_t *>(src) + from, (size_t)m * 2);
                else if (f32)
                    for (int i = 0; i < m; i++) reinterpret_cast<float *>(buf.data())[to + i] = source_value(src, dtype, from + i);
                else
                    for (int i = 0; i < m; i++) reinterpret_cast<uint16_t *>(buf.data())[to + i] = bf16_bits(source_value(src, dtype, from + i));
            }
        unsigned char *d = static_cast<unsigned char *>(dst) + ((size_t)(p.row0 + (r0 / p.rb) * p.rbP * p.row_step) * ld + p.col0) * es;
        IM_CUDA_CHECK(cudaMemcpy2D(d, (size_t)ld * es * p.row_step, buf.data(), (size_t)width * es, (size_t)width * es, n, cudaMemcpyHostToDevice));
    }
    return IM_OK;
}

}  // namespace

// Angles in f64 on the host; the table holds cos and sin of every (position, pair) times the amplitude.
int StackModel::rot_table(const im_stack_layer &c, const float **cosc, const float **sinc) {
    const std::array<double, 8> key = {(double)c.rot_dim, (double)c.rot_dims, c.rot_base, c.yarn_factor, c.yarn_original, c.yarn_fast, c.yarn_slow, c.rot_divide};
    auto it = rot_tables.find(key);
    if (it == rot_tables.end()) {
        const int half = c.rot_dim / 2, n = c.rot_dims / 2, P = cfg.max_seq_len;
        std::vector<double> f((size_t)half, 0.0);
        double amp = 1.0;
        for (int i = 0; i < n; i++) f[i] = pow(c.rot_base, -2.0 * i / c.rot_dims);
        if (c.yarn_factor > 0.0) {  // pairs that turn slowly over the original context are slowed by the factor, fast ones kept
            auto pair_of = [&](double turns) { return c.rot_dims * log(c.yarn_original / (2.0 * M_PI * turns)) / (2.0 * log(c.rot_base)); };
            const double lo = std::max(floor(pair_of(c.yarn_fast)), 0.0), hi = std::min(ceil(pair_of(c.yarn_slow)), c.rot_dims - 1.0);
            for (int i = 0; i < n; i++) {
                const double r = std::min(1.0, std::max(0.0, (i - lo) / std::max(hi - lo, 0.001)));
                f[i] = f[i] / c.yarn_factor * r + f[i] * (1.0 - r);
            }
            amp = 0.1 * log(c.yarn_factor) + 1.0;
        }
        if (c.rot_divide > 0.0)
            for (int i = 0; i < n; i++) f[i] /= c.rot_divide;
        std::vector<float> co((size_t)P * half), si((size_t)P * half);
        for (int p = 0; p < P; p++)
            for (int i = 0; i < half; i++) {
                const double a = (double)p * f[i];
                co[(size_t)p * half + i] = i < n ? (float)(cos(a) * amp) : 1.0f;
                si[(size_t)p * half + i] = i < n ? (float)(sin(a) * amp) : 0.0f;
            }
        float *dc = nullptr, *ds = nullptr;
        IM_TRY(alloc((void **)&dc, co.size() * 4));
        IM_TRY(alloc((void **)&ds, si.size() * 4));
        IM_CUDA_CHECK(cudaMemcpy(dc, co.data(), co.size() * 4, cudaMemcpyHostToDevice));
        IM_CUDA_CHECK(cudaMemcpy(ds, si.data(), si.size() * 4, cudaMemcpyHostToDevice));
        it = rot_tables.emplace(key, std::make_pair(dc, ds)).first;
    }
    *cosc = it->second.first;
    *sinc = it->second.second;
    return IM_OK;
}

int StackModel::load(const std::string &name, const void *data, int dtype, const std::vector<int64_t> &shape) {
    size_t count = 1;
    for (int64_t d : shape) count *= (size_t)d;
    auto expect = [&](int64_t a, int64_t b) -> int {  // b = 0: a vector
        if ((b == 0 && shape.size() == 1 && shape[0] == a) || (b && shape.size() == 2 && shape[0] == a && shape[1] == b)) return IM_OK;
        std::string got;
        for (int64_t d : shape) got += (got.empty() ? "" : ", ") + std::to_string(d);
        return b ? fail(IM_ERR_INVALID, "%s: expected shape [%lld, %lld], got [%s]", name.c_str(), (long long)a, (long long)b, got.c_str())
                 : fail(IM_ERR_INVALID, "%s: expected shape [%lld], got [%s]", name.c_str(), (long long)a, got.c_str());
    };
    // an f32 vector, in padded blocks if bP is given
    auto vec = [&](float **dst, int n, int b = 0, int bP = 0) -> int {
        if (!b) b = bP = n;
        std::vector<float> v((size_t)((n + b - 1) / b) * bP, 0.0f);
        for (int i = 0; i < n; i++) v[(size_t)(i / b) * bP + i % b] = source_value(data, dtype, i);
        IM_TRY(alloc((void **)dst, v.size() * 4));
        IM_CUDA_CHECK(cudaMemcpy(*dst, v.data(), v.size() * 4, cudaMemcpyHostToDevice));
        return IM_OK;
    };
    if (!missing.count(name)) return fail(IM_ERR_INVALID, "tensor '%s' is unknown to this model or was loaded before", name.c_str());
    int rc = IM_ERR_INVALID;
    int l = -1, off = 0;
    if (name == "embed" || name == "head") {
        IM_TRY(expect(sc.vocab, W));
        DenseWeight &w = name == "embed" ? embed : head;
        rc = place(w.w, w.ld, f32, data, dtype, sc.vocab, W, {});
    } else if (name == "embed.norm" || name == "final.norm") {
        IM_TRY(expect(W, 0));
        rc = vec(name == "embed.norm" ? &embed_norm : &final_norm, W);
    } else if (name == "loop.in") {
        IM_TRY(expect(W, 2 * W));
        rc = place(loop_in.w, loop_in.ld, f32, data, dtype, W, 2 * W, {});
    } else if (name == "loop.step") {
        IM_TRY(expect(sc.loop_times, W));
        rc = vec(&loop_step, sc.loop_times * W);
    } else if (sscanf(name.c_str(), "l%d.%n", &l, &off) == 1 && off > 0 && l >= 0 && l < sc.num_layers) {
        StackLayer &L = layers[(size_t)l];
        const im_stack_layer &c = L.c;
        const std::string t = name.substr((size_t)off);
        const bool lat = c.mixer == IM_MIXER_LATENT, lin = L.linear(), grp = c.mixer == IM_MIXER_GROUPED, gat = c.mixer == IM_MIXER_GATED;
        // rows of a per-head projection of the mixer's input
        auto heads_in = [&](int n, int size, int sizeP, int row0) -> int {
            IM_TRY(expect((int64_t)n * size, W));
            Placement p;
            p.rb = size; p.rbP = sizeP;
            p.row0 = row0;
            return place(L.w_in.w, L.w_in.ld, f32, data, dtype, n * size, W, p);
        };
        if (t == "norm1" || t == "norm2") {
            IM_TRY(expect(W, 0));
            rc = vec(t == "norm1" ? &L.norm1 : &L.norm2, W);
        } else if (t == "mlp.gate" || t == "mlp.up") {
            IM_TRY(expect(c.ff, W));
            const DenseWeight &w = post ? L.w_gu : L.w_in;
            Placement p;
            p.row0 = (post ? 0 : L.pair0) + (t == "mlp.up");
            p.row_step = 2;
            rc = place(w.w, w.ld, f32, data, dtype, c.ff, W, p);
        } else if (t == "mlp.down") {
            IM_TRY(expect(W, c.ff));
            const DenseWeight &w = post ? L.w_down : L.w_out;
            Placement p;
            p.col0 = post ? 0 : L.mixP;
            rc = place(w.w, w.ld, f32, data, dtype, W, c.ff, p);
        } else if (t == "mix.o") {
            IM_TRY(expect(W, (int64_t)c.heads * c.vdim));
            Placement p;
            p.cb = c.vdim; p.cbP = L.value_pad();
            rc = place(L.w_out.w, L.w_out.ld, f32, data, dtype, W, c.heads * c.vdim, p);
        } else if (lat && t == "mix.q") {  // per head [dim | rot_dim], each part padded
            IM_TRY(expect((int64_t)c.heads * (c.dim + c.rot_dim), W));
            const size_t es = dtype == IM_DTYPE_F32 ? 4 : 2;
            rc = IM_OK;
            for (int hh = 0; hh < c.heads && rc == IM_OK; hh++) {
                const unsigned char *s = static_cast<const unsigned char *>(data) + (size_t)hh * (c.dim + c.rot_dim) * W * es;
                Placement p;
                p.row0 = L.ls.q_off + hh * (L.ls.dimP + L.ls.rotP);
                rc = place(L.w_in.w, L.w_in.ld, f32, s, dtype, c.dim, W, p);
                p.row0 += L.ls.dimP;
                if (rc == IM_OK) rc = place(L.w_in.w, L.w_in.ld, f32, s + (size_t)c.dim * W * es, dtype, c.rot_dim, W, p);
            }
        } else if (lat && t == "mix.dkv") {
            IM_TRY(expect(c.kv_rank + c.rot_dim, W));
            const size_t es = dtype == IM_DTYPE_F32 ? 4 : 2;
            Placement p;
            p.row0 = L.ls.c_off;
            rc = place(L.w_in.w, L.w_in.ld, f32, data, dtype, c.kv_rank, W, p);
            p.row0 += L.ls.latP;
            if (rc == IM_OK) rc = place(L.w_in.w, L.w_in.ld, f32, static_cast<const unsigned char *>(data) + (size_t)c.kv_rank * W * es, dtype, c.rot_dim, W, p);
        } else if (lat && t == "mix.dkv.norm") {
            IM_TRY(expect(c.kv_rank, 0));
            rc = vec(&L.c_norm, c.kv_rank);
        } else if (lat && (t == "mix.uk" || t == "mix.uv")) {
            const bool k = t == "mix.uk";
            const int d = k ? c.dim : c.vdim;
            IM_TRY(expect((int64_t)c.heads * d, c.kv_rank));
            Placement p;
            p.rb = d; p.rbP = L.ls.dimP + L.ls.vP;
            p.row0 = k ? 0 : L.ls.dimP;
            rc = place(L.ukv, L.ls.latP, f32, data, dtype, c.heads * d, c.kv_rank, p);
        } else if ((lat || grp) && t == "mix.sink") {
            IM_TRY(expect(c.heads, 0));
            rc = vec(&L.sink, c.heads);
        } else if (lin && (t == "mix.q" || t == "mix.k")) {
            rc = heads_in(c.heads, c.dim, L.ns.dimP, t == "mix.q" ? L.ns.q_off : L.ns.k_off);
        } else if (lin && (t == "mix.v" || t == "mix.g")) {
            rc = heads_in(c.heads, c.vdim, L.ns.vP, t == "mix.v" ? L.ns.v_off : L.ns.g_off);
        } else if (lin && t == "mix.norm") {
            const int n = gat ? c.vdim : c.heads * c.vdim;
            IM_TRY(expect(n, 0));
            rc = vec(&L.o_norm, n, c.vdim, L.ns.vP);
        } else if (gat && t == "mix.a1") {
            rc = heads_in(1, c.gate_rank, c.gate_rank, L.f0);
        } else if (gat && t == "mix.a2") {  // kept transposed, [rank, channels]
            const int n = c.heads * c.dim;
            IM_TRY(expect(n, c.gate_rank));
            std::vector<float> v((size_t)n * c.gate_rank);
            for (int i = 0; i < n; i++)
                for (int k = 0; k < c.gate_rank; k++) v[(size_t)k * n + i] = source_value(data, dtype, (size_t)i * c.gate_rank + k);
            IM_TRY(alloc((void **)&L.a2, v.size() * 4));
            IM_CUDA_CHECK(cudaMemcpy(L.a2, v.data(), v.size() * 4, cudaMemcpyHostToDevice));
            rc = IM_OK;
        } else if (gat && t == "mix.a2.b") {
            IM_TRY(expect((int64_t)c.heads * c.dim, 0));
            rc = vec(&L.a2b, c.heads * c.dim);
        } else if (grp && t == "mix.q") {
            rc = heads_in(c.heads, c.dim, L.gs.dimP, L.gs.q_off);
        } else if (grp && t == "mix.k") {
            rc = heads_in(c.kv_heads, c.dim, L.gs.dimP, L.gs.k_off);
        } else if (grp && t == "mix.v") {
            rc = heads_in(c.kv_heads, c.vdim, L.gs.vP, L.gs.v_off);
        } else if (grp && t == "mix.g") {
            rc = heads_in(c.heads, c.vdim, L.gs.vP, L.gs.g_off);
        } else if (grp && (t == "mix.q.norm" || t == "mix.k.norm")) {
            IM_TRY(expect(c.dim, 0));
            rc = vec(t == "mix.q.norm" ? &L.q_norm : &L.k_norm, c.dim);
        } else {
            return fail(IM_ERR_INVALID, "unknown tensor '%s'", name.c_str());
        }
    } else {
        return fail(IM_ERR_INVALID, "unknown tensor '%s'", name.c_str());
    }
    if (rc != IM_OK) return rc;
    missing.erase(name);
    return IM_OK;
}

int StackModel::finalize() {
    if (!missing.empty()) return fail(IM_ERR_STATE, "missing tensor %s (%zu in all)", missing.begin()->c_str(), missing.size());
    const size_t es = elem_size(f32), slots = (size_t)cfg.max_batch, S = (size_t)cfg.max_seq_len;
    bool wide = false, attends = false;  // wide: every token of a prompt chunk keeps its own scratch (absorbed queries, partial sums)
    for (StackLayer &L : layers) {
        const bool lat = L.c.mixer == IM_MIXER_LATENT;
        if (!lat && L.c.mixer != IM_MIXER_GROUPED) continue;
        attends = true;
        if (L.c.rot_dims > 0 || lat) IM_TRY(rot_table(L.c, &L.cosc, &L.sinc));
        if (f32 || !(lat ? latent_expands(L.ls) : grouped_prefills(L.gs))) wide = true;
    }
    if (attends && wide) cfg.prefill_chunk_size = std::min(cfg.prefill_chunk_size, kStackChunkWide);
    MT = std::max(std::max(cfg.max_batch, cfg.prefill_chunk_size), std::min(kAllLogitsChunk, cfg.max_seq_len));
    size_t abs_elems = 0, rec_elems = 0, seg_elems = 0, kv_need = 0, decay_elems = 0;
    int count = 0;
    for (StackLayer &L : layers) {
        ldy = std::max(ldy, L.pair0);
        ldcat = std::max(ldcat, post ? std::max(L.mixP, L.ffP) : L.mixP + L.ffP);
        if (L.c.mixer == IM_MIXER_LATENT) {
            // tokens of one pass in the absorbed form: a decode batch, a short chunk, or (wide) a whole one
            const int one = wide ? MT : std::min(MT, kLatentExpandMin - 1);
            abs_elems = std::max(abs_elems, (size_t)std::max(one, cfg.max_batch) * L.ls.heads * L.ls.rowP);
            for (int t = 1; t <= one; t++) part_bytes = std::max(part_bytes, latent_part_bytes(dev, L.ls, t, 1));
            for (int b = 1; b <= cfg.max_batch; b++) part_bytes = std::max(part_bytes, latent_part_bytes(dev, L.ls, b, b));
            const size_t head_bytes = (size_t)(L.ls.dimP + L.ls.vP) * 2 * S;
            if (!wide) kv_need = std::max(kv_need, std::max(head_bytes, std::min(kExpandBytes, head_bytes * L.ls.heads)));
        } else if (L.c.mixer == IM_MIXER_GROUPED) {
            const int most = std::max(wide ? MT : std::min(MT, kGroupedPrefillMin - 1), cfg.max_batch);
            for (int t = 1; t <= most; t++) part_bytes = std::max(part_bytes, grouped_part_bytes(dev, L.gs, f32, t));
            count = std::max(count, grouped_counters(L.gs, most));
        } else {
            rec_elems = std::max(rec_elems, (size_t)MT * L.ns.heads * L.ns.vP);
            if (L.c.mixer == IM_MIXER_GATED) {
                lda1 = std::max(lda1, round_up(L.ns.rank, 8));
                if (!f32 && MT >= kGatedChunkMin && gated_chunk_takes(L.ns)) {
                    decay_elems = std::max(decay_elems, (size_t)MT * L.ns.heads * L.ns.dimP);
                    chunk_bytes = std::max(chunk_bytes, (size_t)((MT + kGatedChunk - 1) / kGatedChunk) * L.ns.heads * L.ns.dim * L.ns.vS * 4);
                }
            } else if (!f32 && MT >= 2 * kLinearPow) {
                seg_elems = std::max(seg_elems, (size_t)(kLinearSegMax - 1) * L.ns.heads * L.ns.dim * L.ns.vS);
            }
        }
    }
    ldy = std::max(ldy, 8);
    for (StackRun &r : runs) {
        const StackLayer &L = layers[(size_t)r.layer];
        if (L.c.mixer == IM_MIXER_GROUPED) {
            if (L.c.kv_from) {  // the last pass through that layer so far
                for (const StackRun &o : runs) {
                    if (&o == &r) break;
                    if (o.layer == L.c.kv_from - 1) r.cache = o.cache, r.vcache = o.vcache;
                }
                if (!r.cache) return fail(IM_ERR_INVALID, "layer %d: layer %d has not run before it", r.layer, L.c.kv_from - 1);
                continue;
            }
            const size_t rows = slots * S * L.gs.kv_heads * es;
            IM_TRY(alloc(&r.cache, rows * L.gs.dimP));
            IM_TRY(alloc(&r.vcache, rows * L.gs.vP));
            IM_CUDA_CHECK(cudaMemset(r.cache, 0, rows * L.gs.dimP));
            IM_CUDA_CHECK(cudaMemset(r.vcache, 0, rows * L.gs.vP));
            continue;
        }
        const size_t n = L.c.mixer == IM_MIXER_LATENT ? slots * S * L.ls.rowP * es : slots * L.ns.heads * L.ns.dim * L.ns.vS * 4;
        IM_TRY(alloc(&r.cache, n));
        IM_CUDA_CHECK(cudaMemset(r.cache, 0, n));
    }
    for (float **p : {&x, &x_alt, &x0}) IM_TRY(alloc((void **)p, (size_t)MT * W * 4));
    IM_TRY(alloc(&y, (size_t)MT * ldy * es));
    IM_TRY(alloc(&cat, (size_t)MT * ldcat * es));
    IM_TRY(alloc(&h, (size_t)MT * round_up(2 * W, 8) * es));
    IM_CUDA_CHECK(cudaMemset(y, 0, (size_t)MT * ldy * es));
    IM_CUDA_CHECK(cudaMemset(cat, 0, (size_t)MT * ldcat * es));  // padding columns meet zero weights and must be finite
    IM_TRY(alloc(&qabs, abs_elems * es));
    IM_TRY(alloc((void **)&part, part_bytes));
    IM_TRY(alloc(&kv, kv_need));
    kv_bytes = kv_need;
    IM_TRY(alloc((void **)&rec_o, rec_elems * 4));
    IM_TRY(alloc((void **)&seg_sums, seg_elems * 4));
    if (rec_elems) IM_CUDA_CHECK(cudaMemset(rec_o, 0, rec_elems * 4));
    if (post) IM_TRY(alloc((void **)&sub, (size_t)MT * W * 4));
    IM_TRY(alloc((void **)&a1, (size_t)MT * lda1 * 4));
    IM_TRY(alloc((void **)&decays, decay_elems * 4));
    IM_TRY(alloc((void **)&chunk_states, chunk_bytes));
    IM_TRY(alloc((void **)&counters, (size_t)count * 4));
    if (count) IM_CUDA_CHECK(cudaMemset(counters, 0, (size_t)count * 4));
    IM_TRY(alloc((void **)&logits, slots * cfg.vocab_size * 4));
    logits_dev = logits;
    IM_TRY(session_alloc(this));
    IM_TRY(dense_prepare(dev));
    IM_TRY(latent_prepare(dev));
    IM_TRY(linear_prepare(dev));
    IM_TRY(grouped_prepare(dev));
    IM_CUDA_CHECK(cudaDeviceSynchronize());
    return IM_OK;
}

// cap tanh(head rms(x) g / cap) of n consecutive rows of the residual, from `row` on.  src: the residual, a sublayer's output that
// is still to be added included; leaves its rows in last_x.
int StackModel::logits_of(DenseSrc src, int row, int n, float *out, cudaStream_t st, int *nl) {
    const size_t off = (size_t)row * W;
    src.xf += off;
    last_x = src.xf;
    last_rows = n;
    if (src.kind == kSrcAddNorm) {
        src.xf2 += off;
        src.xout += off;
        src.gamma2 = final_norm;
        last_x = src.xout;
    } else {
        src.kind = kSrcNorm;
        src.gamma = final_norm;
    }
    DenseEpi e;
    e.kind = kEpiF32; e.xf = out; e.ldx = cfg.vocab_size; e.cap = sc.logit_softcap;
    *nl += dense_launches(n, W, src.kind);
    return dense_project(dev, sc.tied_head ? embed : head, src, e, n, h, st);
}

// The mixer of a run: projected rows in y (and a1), heads to cat.
int StackModel::mix(const StackRun &r, int nseq, int T, const int *slots, cudaStream_t st, int *nl) {
    const StackLayer &L = layers[(size_t)r.layer];
    const int host_pos = prefill_slot_id >= 0 ? prefill_ctx_begin : -1, splits_ctx = prefill_slot_id >= 0 ? prefill_ctx_end : cfg.max_seq_len;
    if (L.c.mixer == IM_MIXER_LATENT) {
        LatentArgs a{};
        a.s = L.ls; a.f32 = f32; a.y = y; a.ldy = ldy; a.ukv = L.ukv; a.uk_ld = L.ls.latP; a.c_norm = L.c_norm; a.sink = L.sink;
        a.cosc = L.cosc; a.sinc = L.sinc; a.cache = r.cache; a.max_seq = cfg.max_seq_len; a.nseq = nseq; a.T = T; a.pos_dev = pos_dev; a.slot_map = slots;
        a.out = cat; a.ldo = ldcat; a.qabs = qabs; a.part = part; a.part_bytes = part_bytes; a.kv = kv; a.kv_bytes = kv_bytes;
        a.host_slot = prefill_slot_id; a.host_pos = host_pos; a.splits_ctx = splits_ctx;
        return latent_attention_run(dev, a, st, nl);
    }
    if (L.c.mixer == IM_MIXER_GROUPED) {
        GroupedArgs a{};
        a.s = L.gs; a.f32 = f32; a.y = y; a.ldy = ldy; a.q_norm = L.q_norm; a.k_norm = L.k_norm; a.sink = L.sink; a.cosc = L.cosc; a.sinc = L.sinc;
        a.kcache = r.cache; a.vcache = r.vcache; a.max_seq = cfg.max_seq_len; a.nseq = nseq; a.T = T; a.pos_dev = pos_dev; a.slot_map = slots;
        a.out = cat; a.ldo = ldcat; a.part = part; a.part_bytes = part_bytes; a.counters = counters;
        a.host_slot = prefill_slot_id; a.host_pos = host_pos; a.splits_ctx = splits_ctx;
        return grouped_attention_run(dev, a, st, nl);
    }
    LinearArgs a{};
    a.s = L.ns; a.f32 = f32; a.y = y; a.ldy = ldy; a.norm = L.o_norm; a.pows = L.pows; a.state = static_cast<float *>(r.cache);
    a.a1 = a1; a.a2 = L.a2; a.a2b = L.a2b; a.decays = decays; a.chunk_states = chunk_states; a.chunk_bytes = chunk_bytes;
    a.nseq = nseq; a.T = T; a.pos_dev = pos_dev; a.slot_map = slots; a.keep_state = uncounted ? 1 : 0; a.o = rec_o; a.seg_sums = seg_sums; a.out = cat; a.ldo = ldcat;
    return linear_attention_run(dev, a, st, nl);
}

int StackModel::forward(int nseq, int T, cudaStream_t st, int *launches, Prof *prof, bool all_logits, const int *slots) {
    const int M = nseq * T;
    int nl = 1;
    IM_TRY(stack_embed(tokens_dev, embed.w, f32, embed.ld, embed_norm, sc.embed_scale, x, x0, W, (uint32_t)sc.vocab, sc.norm_eps, M, st));
    IM_MARK(kCatEmbed);
    float *cur = x, *other = x_alt;
    DenseSrc res;  // how the next reader gets the residual (post-norm: with the last sublayer's output still in `sub`)
    res.ldx = W; res.width = W; res.eps = sc.norm_eps; res.xf = cur;
    res.kind = post ? kSrcAddNorm : kSrcNorm;
    auto read_residual = [&](const DenseWeight &w, const DenseEpi &e) -> int {
        IM_TRY(dense_project(dev, w, res, e, M, h, st));
        nl += dense_launches(M, w.K, res.kind);
        if (res.xf2) {  // the sum has been written to `other`
            std::swap(cur, other);
            res.xf = cur; res.xf2 = nullptr; res.gamma = nullptr; res.xout = nullptr;
        }
        return IM_OK;
    };
    auto sublayer_out = [&](const DenseWeight &w, const float *gamma) -> int {
        DenseSrc s;
        s.x = cat; s.ldx = ldcat;
        DenseEpi e;
        e.kind = post ? kEpiF32 : kEpiResidual; e.xf = post ? sub : cur; e.ldx = W;
        IM_TRY(dense_project(dev, w, s, e, M, nullptr, st));
        nl += dense_launches(M, w.K, s.kind);
        if (post) {
            res.xf2 = sub; res.gamma = gamma; res.xout = other;
        }
        return IM_OK;
    };
    for (const StackRun &r : runs) {
        const StackLayer &L = layers[(size_t)r.layer];
        if (r.opens) {
            DenseSrc s;
            s.kind = kSrcConcat; s.xf = cur; s.xf2 = x0; s.ldx = W; s.width = W;
            DenseEpi e;
            e.kind = kEpiF32; e.xf = other; e.ldx = W; e.bias = loop_step + (size_t)r.pass * W;
            IM_TRY(dense_project(dev, loop_in, s, e, M, h, st));
            nl += dense_launches(M, 2 * W, s.kind);
            std::swap(cur, other);
            res.xf = cur;
            IM_MARK(kCatResNorm);
        }
        DenseEpi e;
        e.kind = kEpiProj; e.y = y; e.ldy = ldy; e.silu_end = L.silu_end; e.pair0 = L.pair0; e.pair_silu = sc.ff_act == IM_ACT_SILU;
        e.f0 = L.f0; e.xf = a1; e.ldx = L.linear() ? round_up(L.ns.rank, 8) : 0;
        e.act = static_cast<unsigned char *>(cat) + (size_t)(post ? 0 : L.mixP) * elem_size(f32);
        e.ldact = ldcat;
        if (!post) res.gamma = L.norm1;
        IM_TRY(read_residual(L.w_in, e));
        IM_MARK(kCatQkv);
        IM_TRY(mix(r, nseq, T, slots, st, &nl));
        IM_MARK(kCatAttn);
        IM_TRY(sublayer_out(L.w_out, L.norm1));
        IM_MARK(post ? kCatOProj : kCatDown);
        if (post && L.c.ff > 0) {
            e.silu_end = e.pair0 = 0;
            e.f0 = 1 << 30;
            IM_TRY(read_residual(L.w_gu, e));
            IM_MARK(kCatFfn);
            IM_TRY(sublayer_out(L.w_down, L.norm2));
            IM_MARK(kCatDown);
        }
    }
    if (all_logits) {
        IM_TRY(logits_of(res, 0, M, rows, st, &nl));
    } else if (T == 1) {
        IM_TRY(logits_of(res, 0, M, logits, st, &nl));
    } else {
        for (int s = 0; s < nseq; s++) IM_TRY(logits_of(res, s * T + T - 1, 1, logits + (size_t)s * cfg.vocab_size, st, &nl));
    }
    IM_MARK(kCatHead);
    if (launches) *launches = nl;
    return IM_OK;
}

int StackModel::hidden_rows(int n, float *out_host) {
    if (!last_x || n > last_rows) return fail(IM_ERR_BOUNDS, "the last step left %d rows, %d asked for", last_rows, n);
    if (!hidden) IM_TRY(alloc((void **)&hidden, (size_t)MT * W * 4));
    IM_CUDA_CHECK(launch_k(rms_rows_kernel, dim3(n), dim3(256), 0, stream, last_x, (const float *)final_norm, hidden, W, sc.norm_eps));
    IM_CUDA_CHECK(cudaMemcpyAsync(out_host, hidden, (size_t)n * W * 4, cudaMemcpyDeviceToHost, stream));
    IM_CUDA_CHECK(cudaStreamSynchronize(stream));
    return IM_OK;
}

size_t StackModel::step_bytes(int ctx, int batch) const {
    const size_t es = elem_size(f32);
    size_t b = (size_t)sc.vocab * W * es + (size_t)batch * W * es;
    for (const StackRun &r : runs) {
        const StackLayer &L = layers[(size_t)r.layer];
        const im_stack_layer &c = L.c;
        size_t n = (size_t)W * 3 * c.ff + (size_t)W * c.heads * c.vdim;
        if (c.mixer == IM_MIXER_LATENT)
            n += (size_t)W * ((size_t)c.heads * (c.dim + c.rot_dim) + c.kv_rank + c.rot_dim) + (size_t)c.heads * (c.dim + c.vdim) * c.kv_rank +
                 (size_t)batch * ctx * (c.kv_rank + c.rot_dim);
        else if (c.mixer == IM_MIXER_GROUPED)
            n += (size_t)W * (c.heads * (c.dim + c.vdim) + (c.kv_from ? 0 : c.kv_heads * (c.dim + c.vdim))) +
                 (size_t)batch * (c.chunk ? std::min(ctx, c.chunk) : ctx) * c.kv_heads * (c.dim + c.vdim);
        else
            n += (size_t)W * (2 * c.heads * (c.dim + c.vdim) + (c.mixer == IM_MIXER_GATED ? c.gate_rank : 0));
        b += n * es;
        if (L.linear()) b += (size_t)batch * c.heads * c.dim * c.vdim * 8;  // state read and written
        if (c.mixer == IM_MIXER_GATED) b += (size_t)c.heads * c.dim * (c.gate_rank + 1) * 4;
        if (r.opens) b += (size_t)2 * W * W * es;
    }
    return b;
}

static int stack_plan(StackModel *m, const im_stack_config &c) {
    const int W = c.width;
    for (const char *n : {"embed", "final.norm"}) m->missing.insert(n);
    if (c.embed_scale == 0.0f) m->missing.insert("embed.norm");
    if (c.loop_times > 0) {
        m->missing.insert("loop.in");
        m->missing.insert("loop.step");
        IM_TRY(m->dense_alloc(&m->loop_in, W, 2 * W));
    }
    IM_TRY(m->dense_alloc(&m->embed, c.vocab, W));
    if (!c.tied_head) {
        m->missing.insert("head");
        IM_TRY(m->dense_alloc(&m->head, c.vocab, W));
    }
    for (int i = 0; i < c.num_layers; i++) {
        StackLayer &L = m->layers[(size_t)i];
        const im_stack_layer &q = L.c;
        auto need = [&](const char *t) { m->missing.insert("l" + std::to_string(i) + "." + t); };
        need("norm1");
        if (q.mixer == IM_MIXER_LATENT) {
            LatentShape &s = L.ls;
            s.heads = q.heads; s.dim = q.dim; s.rot_dim = q.rot_dim; s.vdim = q.vdim; s.kv_rank = q.kv_rank; s.scale = q.scale; s.eps = c.norm_eps;
            latent_layout(&s);
            L.pair0 = s.c_off + s.latP + s.rotP;
            L.mixP = s.heads * s.vP;
            for (const char *t : {"mix.q", "mix.dkv", "mix.dkv.norm", "mix.uk", "mix.uv", "mix.sink", "mix.o"}) need(t);
            const size_t n = (size_t)s.heads * (s.dimP + s.vP) * s.latP * elem_size(m->f32);
            IM_TRY(m->alloc(&L.ukv, n));
            IM_CUDA_CHECK(cudaMemset(L.ukv, 0, n));
        } else if (q.mixer == IM_MIXER_GROUPED) {
            GroupedShape &s = L.gs;
            s.heads = q.heads; s.kv_heads = q.kv_heads; s.dim = q.dim; s.vdim = q.vdim; s.rot_dims = q.rot_dims; s.chunk = q.chunk; s.scale = q.scale; s.eps = c.norm_eps;
            grouped_layout(&s, q.kv_from == 0);
            L.pair0 = s.g_off + s.heads * s.vP;
            L.mixP = s.heads * s.vP;
            for (const char *t : {"mix.q", "mix.q.norm", "mix.sink", "mix.g", "mix.o"}) need(t);
            if (!q.kv_from)
                for (const char *t : {"mix.k", "mix.v", "mix.k.norm"}) need(t);
        } else {
            m->has_state = true;
            LinearShape &s = L.ns;
            s.heads = q.heads; s.dim = q.dim; s.vdim = q.vdim; s.eps = c.norm_eps;
            s.dimP = round_up(q.dim, 8); s.vP = round_up(q.vdim, 8); s.vS = round_up(q.vdim, 4);
            s.q_off = 0; s.k_off = s.heads * s.dimP; s.v_off = 2 * s.k_off; s.g_off = s.v_off + s.heads * s.vP;
            L.pair0 = s.g_off + s.heads * s.vP;
            L.mixP = s.heads * s.vP;
            for (const char *t : {"mix.q", "mix.k", "mix.v", "mix.g", "mix.o", "mix.norm"}) need(t);
            if (q.mixer == IM_MIXER_GATED) {
                s.gated = 1; s.rank = q.gate_rank; s.inv_tau = 1.0f / q.tau; s.q_scale = (float)(1.0 / sqrt((double)q.dim));
                L.f0 = L.pair0;
                L.pair0 += round_up(s.rank, 8);
                for (const char *t : {"mix.a1", "mix.a2", "mix.a2.b"}) need(t);
            } else {
                L.silu_end = s.g_off;
                std::vector<float> pw((size_t)s.heads * (kLinearPow + 1));
                for (int hh = 0; hh < s.heads; hh++)
                    for (int n = 0; n <= kLinearPow; n++) pw[(size_t)hh * (kLinearPow + 1) + n] = (float)pow(L.decay[(size_t)hh], n);
                IM_TRY(m->alloc((void **)&L.pows, pw.size() * 4));
                IM_CUDA_CHECK(cudaMemcpy(L.pows, pw.data(), pw.size() * 4, cudaMemcpyHostToDevice));
            }
        }
        L.ffP = round_up(q.ff, 8);
        if (q.ff > 0)
            for (const char *t : {"mlp.gate", "mlp.up", "mlp.down"}) need(t);
        IM_TRY(m->dense_alloc(&L.w_in, L.pair0 + (m->post ? 0 : 2 * q.ff), W));
        IM_TRY(m->dense_alloc(&L.w_out, W, L.mixP + (m->post ? 0 : L.ffP)));
        if (m->post && q.ff > 0) {
            need("norm2");
            IM_TRY(m->dense_alloc(&L.w_gu, 2 * q.ff, W));
            IM_TRY(m->dense_alloc(&L.w_down, W, L.ffP));
        }
    }
    for (int i = 0; i < c.num_layers; i++) {
        if (c.loop_times > 0 && i == c.loop_start) {
            for (int t = 0; t < c.loop_times; t++)
                for (int j = c.loop_start; j < c.loop_stop; j++) {
                    StackRun r;
                    r.layer = j; r.pass = t; r.opens = j == c.loop_start;
                    m->runs.push_back(r);
                }
            i = c.loop_stop - 1;
            continue;
        }
        StackRun r;
        r.layer = i;
        m->runs.push_back(r);
    }
    return IM_OK;
}

}  // namespace im

using namespace im;

IM_EXPORT int im_cuda_model_create_stack(im_device *dev, const im_stack_config *cfg, im_model **out) {
    IM_GUARD_BEGIN
    IM_REQUIRE(dev && cfg && out, "bad argument");
    *out = nullptr;
    im_stack_config c = *cfg;
    if (c.max_seq_len == 0) c.max_seq_len = 2048;
    if (c.max_batch == 0) c.max_batch = 1;
    if (c.prefill_chunk_size == 0) c.prefill_chunk_size = kStackChunk;
    IM_REQUIRE(c.vocab > 0 && c.width > 0 && c.num_layers > 0 && c.layers, "vocab, width and the list of layers must not be empty");
    IM_REQUIRE(c.max_seq_len > 0 && c.max_batch >= 1 && c.max_batch <= kMaxSlots, "max_seq_len must be > 0 and max_batch in 1..%d", kMaxSlots);
    IM_REQUIRE(c.prefill_chunk_size > 0 && c.prefill_chunk_size <= kStackChunk, "prefill_chunk_size must be in 0..%d", kStackChunk);
    IM_REQUIRE(c.norm_eps >= 0.0f && c.logit_softcap >= 0.0f, "norm_eps and logit_softcap must not be negative");
    IM_REQUIRE((c.block == IM_BLOCK_PARALLEL || c.block == IM_BLOCK_POSTNORM) && (c.ff_act == IM_ACT_GELU_TANH || c.ff_act == IM_ACT_SILU), "unknown block or activation");
    IM_REQUIRE(c.block == IM_BLOCK_PARALLEL || c.loop_times == 0, "post-norm blocks are not looped");
    IM_REQUIRE(c.loop_times == 0 || (c.loop_times > 0 && c.loop_start >= 0 && c.loop_start < c.loop_stop && c.loop_stop <= c.num_layers),
               "bad loop %d .. %d x %d over %d layers", c.loop_start, c.loop_stop, c.loop_times, c.num_layers);
    for (int i = 0; i < c.num_layers; i++) {
        const im_stack_layer &q = c.layers[i];
        IM_REQUIRE(q.heads > 0 && q.dim > 0 && q.vdim > 0 && q.ff >= 0, "layer %d: sizes must be positive", i);
        if (q.mixer == IM_MIXER_LATENT) {
            IM_REQUIRE(q.kv_rank > 0 && q.kv_rank <= 1024 && q.rot_dim >= 0 && q.rot_dim % 2 == 0 && q.rot_dims % 2 == 0 && q.rot_dims >= 0 && q.rot_dims <= q.rot_dim,
                       "layer %d: kv_rank must be in 1..1024, rot_dim and the rotated size even, the latter not the larger", i);
            IM_REQUIRE(q.rot_dims == 0 || (q.rot_base > 0.0 && (q.yarn_factor == 0.0 || (q.yarn_factor > 0.0 && q.yarn_original > 0.0 && q.yarn_fast > 0.0 &&
                                                                                        q.yarn_slow > 0.0 && q.rot_base != 1.0))),
                       "layer %d: bad rotation constants", i);
        } else if (q.mixer == IM_MIXER_LINEAR) {
            IM_REQUIRE(q.decay_host && q.dim <= 512, "layer %d: linear attention needs its decays and a key size of at most 512", i);
        } else if (q.mixer == IM_MIXER_GATED) {
            IM_REQUIRE(q.gate_rank > 0 && q.tau > 0.0f && q.dim <= 512, "layer %d: gated linear attention needs a gate of rank > 0, tau > 0 and a key size of at most 512", i);
        } else if (q.mixer == IM_MIXER_GROUPED) {
            IM_REQUIRE(q.kv_heads > 0 && q.heads % q.kv_heads == 0, "layer %d: %d query heads do not share %d key / value heads evenly", i, q.heads, q.kv_heads);
            IM_REQUIRE(q.vdim <= 1024 && q.chunk >= 0 && q.rot_dims >= 0 && q.rot_dims % 2 == 0 && q.rot_dims <= q.dim && q.rot_dim == q.rot_dims,
                       "layer %d: value sizes are at most 1024, the rotated size is even and at most the head's", i);
            IM_REQUIRE(q.rot_dims == 0 || (q.rot_base > 0.0 && q.rot_divide >= 0.0 && q.yarn_factor == 0.0), "layer %d: bad rotation constants", i);
            if (q.kv_from) {
                IM_REQUIRE(q.kv_from > 0 && q.kv_from <= i, "layer %d: keys and values come from an earlier layer", i);
                const im_stack_layer &o = c.layers[q.kv_from - 1];
                IM_REQUIRE(o.mixer == IM_MIXER_GROUPED && o.kv_from == 0 && o.kv_heads == q.kv_heads && o.dim == q.dim && o.vdim == q.vdim,
                           "layer %d: layer %d has no keys and values of this shape", i, q.kv_from - 1);
            }
        } else {
            return fail(IM_ERR_INVALID, "layer %d: unknown mixer %d", i, q.mixer);
        }
    }
    IM_CUDA_CHECK(cudaSetDevice(dev->ordinal));
    StackModel *m = new StackModel();
    m->dev = dev;
    m->f32 = c.compute_f32 ? 1 : 0;
    m->W = c.width;
    m->post = c.block == IM_BLOCK_POSTNORM;
    m->layers.resize((size_t)c.num_layers);
    for (int i = 0; i < c.num_layers; i++) {
        m->layers[(size_t)i].c = c.layers[i];
        if (c.layers[i].mixer == IM_MIXER_LINEAR) m->layers[(size_t)i].decay.assign(c.layers[i].decay_host, c.layers[i].decay_host + c.layers[i].heads);
        m->layers[(size_t)i].c.decay_host = nullptr;
    }
    c.layers = nullptr;
    m->sc = c;
    im_model_config &g = m->cfg;  // the fields the session reads
    g.num_layers = c.num_layers; g.hidden_size = c.width; g.vocab_size = c.vocab; g.max_seq_len = c.max_seq_len; g.max_batch = c.max_batch;
    g.rms_eps = c.norm_eps; g.tp_world = 1; g.prefill_chunk_size = std::min(c.prefill_chunk_size, c.max_seq_len);
    m->logits_f32 = 1;
    int rc = session_open(m);
    if (rc == IM_OK) rc = stack_plan(m, c);
    if (rc != IM_OK) {
        const std::string why = last_error();
        im_cuda_model_free(m);
        last_error() = why;
        return rc;
    }
    *out = m;
    return IM_OK;
    IM_GUARD_END
}

IM_EXPORT int im_cuda_model_load_tensor(im_model *h, const char *name, const void *data_host, int dtype, int ndim, const int64_t *shape) {
    IM_GUARD_BEGIN
    IM_REQUIRE(h && name && data_host && shape && ndim >= 1, "bad argument");
    IM_REQUIRE(dtype == IM_DTYPE_F16 || dtype == IM_DTYPE_F32 || dtype == IM_DTYPE_BF16, "unknown element type %d", dtype);
    StackModel *m = dynamic_cast<StackModel *>(h);
    if (!m) return fail(IM_ERR_INVALID, "this call is for models given as a list of layers, the model is of family '%s'", h->family());
    if (m->finalized) return fail(IM_ERR_STATE, "model already finalized");
    IM_CUDA_CHECK(cudaSetDevice(m->dev->ordinal));
    return m->load(name, data_host, dtype, std::vector<int64_t>(shape, shape + ndim));
    IM_GUARD_END
}
