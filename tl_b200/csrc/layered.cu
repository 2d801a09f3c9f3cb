// A decoder described as a list of layers (model_desc.h), each with one of several mixers and an optional feed-forward: weights
// stacked per launch, caches and recurrent state per sequence, and the three ways a session runs it.
//   one token      norm -> stacked input projections | mixer | output projection | norm -> up | activation -> down, chained with
//                  programmatic dependent launch; what a sublayer leaves joins the residual in its last launch, or - where it is
//                  gated and normed first - in the prologue of the next sublayer's first launch
//   one token of every sequence of a batch, and T tokens of one sequence: the same steps over rows, linear layers as GEMMs
// The residual, norms, routers, scores, recurrences and everything that enters them stay in 32-bit floats.
#include "model_desc.h"

#include <algorithm>
#include <cmath>

#include "layered_kernels.h"

namespace tlb {

namespace {

struct Layer {
    const LayerDesc *d = nullptr;
    DenseW in, o, up, down, w2;
    DenseW uq, uk, uv, uk16, uv16;         // latent attention
    DenseW eup, edown, sdown;              // experts, stacked (w.n rows each); shared expert's second matrix
    RouteDesc route;
    tlb_tensor *norm1 = nullptr, *norm2 = nullptr, *post1 = nullptr, *post2 = nullptr, *ls1 = nullptr, *ls2 = nullptr, *act = nullptr;
    tlb_tensor *sink = nullptr, *onorm = nullptr, *w0 = nullptr, *qnorm = nullptr, *cnorm = nullptr;
    // columns of the stacked projections (-1: absent), those of `up` behind its gated activations
    int c_kv = -1, c_gate = -1, c_rg1 = -1, u_rg2 = -1, u_router = -1, u_sg = -1;
    uint64_t step_bytes = 0;               // weights one decoded token reads
    float *bias = nullptr;                 // by distance, [heads][bias_n]
    int bias_n = 0;
    float *decay = nullptr, *rot_cos = nullptr, *rot_sin = nullptr;
    void *kcache = nullptr, *vcache = nullptr;
    float *state = nullptr;
    int out_width = 0;                     // columns the output projection reads
};

struct RotTable { int dims; double base; RotScaling scaling; float *cos_t, *sin_t; };

// Work rows of a pass over T rows.
struct RowBufs {
    float *x = nullptr, *proj = nullptr, *u = nullptr, *o = nullptr, *y = nullptr, *q = nullptr, *dly = nullptr;
    float2 *look = nullptr;
    void *act = nullptr, *hid = nullptr, *th = nullptr;
    // mixture of experts: T * top rows
    MoePlan plan;
    float *yp = nullptr, *ysh = nullptr;
    void *xp = nullptr, *hp = nullptr;
    // latent attention, rows of queries in the latent space
    void *qa = nullptr;
    float *partial = nullptr;
};
// Whose rows they are: one new token of every sequence (pos, rope on the device), or tokens of one sequence.
struct RowCtx {
    int T = 0, seq = 0, pos0 = 0, rope0 = 0, rope_step = 0;
    const int *pos = nullptr, *rope = nullptr;
};

}  // namespace

struct LayeredModel {
    ModelDesc desc;
    LayeredCfg cfg;
    std::vector<Layer> layers;
    DenseW head;
    const __nv_bfloat16 *embed = nullptr;
    int embed_ld = 0;
    tlb_tensor *final_norm = nullptr;
    std::vector<tlb_tensor *> held;        // tensors of the map the session keeps alive
    std::vector<Storage *> stores;
    std::vector<RotTable> rots;
    RowBufs batch_rows;                    // of a session with several sequences (x: the session's)
    // one token: projections (a layer's residual gate is read while the next layer writes: two), mixer output, up projection
    float *proj[2] = {nullptr, nullptr}, *mix = nullptr, *up = nullptr, *partial = nullptr;
    float *x2 = nullptr, *y = nullptr, *h = nullptr, *q = nullptr, *hid = nullptr, *ex = nullptr, *weight = nullptr;
    void *qa = nullptr;
    int *counters = nullptr, *sel = nullptr;
    int ldp = 0, ldm = 0, ldu = 0, lda = 0, ldq = 0;
    uint64_t weight_bytes = 0;
};

namespace {

template <typename T>
tlb_status alloc(LayeredModel *lm, T **p, size_t count, bool zero = true)
{
    Storage *s = storage_alloc(count * sizeof(T));
    if (!s) return TLB_ERR_ALLOC;
    lm->stores.push_back(s);
    *p = (T *)s->ptr;
    if (zero) TLB_CUDA(cudaMemsetAsync(s->ptr, 0, count * sizeof(T), ctx()->stream));
    return TLB_OK;
}

// proj: the first projection's rows, q: the queries' (in proj where they are projected directly)
MixLatent latent_args(const LayeredModel *lm, const Layer &L, const float *proj, int ldp, float *q, int ldq)
{
    const MixerDesc &x = L.d->mix;
    MixLatent m = {};
    m.H = x.heads; m.D = x.dim; m.RD = x.rot_dim; m.DV = x.vdim; m.R = x.kv_rank; m.ld = latent_ld(x.kv_rank, x.rot_dim);
    m.max_seq = lm->cfg.max_seq; m.window = std::min(x.window > 0 ? x.window : lm->cfg.max_seq, lm->cfg.max_seq);
    m.scale = x.scale; m.eps = lm->desc.eps; m.rot = x.rot_dims; m.rot_cos = L.rot_cos; m.rot_sin = L.rot_sin;
    m.c_norm = L.cnorm ? L.cnorm->f32() : nullptr; m.uk = L.uk; m.uv = L.uv; m.uk16 = L.uk16; m.uv16 = L.uv16;
    m.cache = L.kcache; m.seq_stride = (size_t)lm->cfg.max_seq * m.ld;
    m.q = x.q_rank ? q : const_cast<float *>(proj); m.ldq = x.q_rank ? ldq : ldp;
    m.kv = proj ? proj + L.c_kv : nullptr; m.ldkv = ldp;
    m.gate = proj && L.c_gate >= 0 ? proj + L.c_gate : nullptr; m.ld_gate = ldp;
    return m;
}

struct Loader {
    LayeredModel *lm;
    tlb_map *m;

    tlb_status matrix(const std::string &name, const tlb_tensor **t, int64_t n, int64_t k)
    {
        *t = map_raw_bf16(m, name);
        if (!*t) return map_has(m, name) ? fail(TLB_ERR_TYPE, "tensor '%s' is not bf16", name.c_str()) : fail(TLB_ERR_ARG, "Tensor '%s' not found in map", name.c_str());
        if ((*t)->rank != 2 || ((n >= 0) && (*t)->shape[0] != n) || (*t)->shape[1] != k)
            return fail(TLB_ERR_SHAPE, "tensor '%s' is not [%lld, %lld]", name.c_str(), (long long)n, (long long)k);
        lm->weight_bytes += (uint64_t)(*t)->numel() * 2;
        return TLB_OK;
    }
    tlb_status vec(const std::string &name, tlb_tensor **t, int64_t n)
    {
        TLB_TRY(tlb_map_get(t, m, name.c_str()));
        lm->held.push_back(*t);
        if ((*t)->numel() != n) return fail(TLB_ERR_SHAPE, "tensor '%s' has %lld elements, expected %lld", name.c_str(), (long long)(*t)->numel(), (long long)n);
        lm->weight_bytes += (uint64_t)n * 4;
        return TLB_OK;
    }
    // several [n_i, k] matrices as one, rows one after the other; a single matrix whose rows are whole 16-byte lines stays where it is
    struct Part { std::string name; int n; bool bias; };
    // the two [ff, k] matrices of a gated activation; they come first, in pairs (DenseW::glu)
    struct Glu { std::string gate, up; int ff; };
    static int glu_rows(int ff) { return 2 * ((ff + 1) / 2 * 2); }
    tlb_status stack(DenseW *w, const std::vector<Part> &parts, int k, const std::vector<Glu> &pairs = {}, int act = 0)
    {
        int n = 0, glu = 0;
        bool any_bias = false;
        for (const Glu &g : pairs) glu += glu_rows(g.ff);
        for (const Part &p : parts) { n += p.n; any_bias |= p.bias; }
        n += glu;
        w->n = n; w->k = k; w->ld = act_ld(k); w->glu = glu; w->glu_act = act;
        if (parts.size() == 1 && !glu && w->ld == k) {
            const tlb_tensor *t;
            TLB_TRY(matrix(parts[0].name, &t, n, k));
            tlb_tensor_retain(const_cast<tlb_tensor *>(t));
            lm->held.push_back(const_cast<tlb_tensor *>(t));
            w->w = (const __nv_bfloat16 *)t->data();
        } else {
            __nv_bfloat16 *dst;
            bool odd = false;
            for (const Glu &g : pairs) odd |= g.ff % 2 != 0;
            TLB_TRY(alloc(lm, &dst, (size_t)n * w->ld, w->ld != k || odd));
            int at = 0;
            for (const Glu &g : pairs) {
                for (int up = 0; up < 2; up++) {
                    const tlb_tensor *t;
                    TLB_TRY(matrix(up ? g.up : g.gate, &t, g.ff, k));
                    TLB_TRY(launch_pack_glu_rows((const __nv_bfloat16 *)t->data(), g.ff, k, dst + (size_t)at * w->ld, w->ld, up));
                }
                at += glu_rows(g.ff);
            }
            for (const Part &p : parts) {
                const tlb_tensor *t;
                TLB_TRY(matrix(p.name, &t, p.n, k));
                TLB_TRY(launch_pack_rows((const __nv_bfloat16 *)t->data(), p.n, k, dst + (size_t)at * w->ld, w->ld, 0));
                at += p.n;
            }
            w->w = dst;
        }
        if (any_bias) {
            float *b;
            TLB_TRY(alloc(lm, &b, n));
            int at = glu;
            for (const Part &p : parts) {
                if (p.bias) {
                    tlb_tensor *t;
                    TLB_TRY(vec(p.name + ".b", &t, p.n));
                    TLB_CUDA(cudaMemcpyAsync(b + at, t->data(), (size_t)p.n * 4, cudaMemcpyDeviceToDevice, ctx()->stream));
                }
                at += p.n;
            }
            w->bias = b;
        }
        return TLB_OK;
    }
    // a matrix again with its values as f16, for GEMMs over f16 rows
    tlb_status as_f16(DenseW *dst, const std::string &name, int n, int k)
    {
        const tlb_tensor *t;
        const uint64_t before = lm->weight_bytes;
        TLB_TRY(matrix(name, &t, n, k));
        lm->weight_bytes = before;
        __half *p;
        *dst = DenseW();
        dst->n = n; dst->k = k; dst->ld = act_ld(k); dst->f16 = true;
        TLB_TRY(alloc(lm, &p, (size_t)n * dst->ld, false));
        dst->w = (const __nv_bfloat16 *)p;
        return launch_pack_rows_f16((const __nv_bfloat16 *)t->data(), n, k, p, dst->ld);
    }
    tlb_status upload(float **dst, const std::vector<float> &v)
    {
        TLB_TRY(alloc(lm, dst, v.size(), false));
        TLB_CUDA(cudaMemcpyAsync(*dst, v.data(), v.size() * 4, cudaMemcpyHostToDevice, ctx()->stream));
        TLB_CUDA(cudaStreamSynchronize(ctx()->stream));
        return TLB_OK;
    }
    tlb_status host(const tlb_tensor *t, std::vector<float> *v)
    {
        v->resize((size_t)t->numel());
        return tlb_tensor_to_host(t, v->data(), v->size() * 4);
    }

    // cos / sin of the angles of every position, in double.  With scaling, pairs that turn seldom within the original length are
    // slowed down by the factor (a ramp between the two bounds on turns), and both tables grow by 0.1 ln(factor) + 1.
    tlb_status rotation(int dims, double base, const RotScaling &sc, float **c, float **s)
    {
        for (const RotTable &r : lm->rots)
            if (r.dims == dims && r.base == base && r.scaling == sc) { *c = r.cos_t; *s = r.sin_t; return TLB_OK; }
        const int half = dims / 2, n = lm->cfg.max_seq;
        const double pi = 3.14159265358979323846;
        double lo = 0.0, hi = 0.0, gain = 1.0;
        if (sc.factor > 0.0) {
            auto pair_of = [&](double turns) { return dims * std::log(sc.original / (2.0 * pi * turns)) / (2.0 * std::log(base)); };
            lo = std::max(std::floor(pair_of(sc.fast)), 0.0);
            hi = std::min(std::ceil(pair_of(sc.slow)), (double)dims - 1.0);
            gain = 0.1 * std::log(sc.factor) + 1.0;
        }
        std::vector<float> hc((size_t)n * half), hs((size_t)n * half);
        for (int i = 0; i < half; i++) {
            double f = std::pow(base, -2.0 * i / dims);
            if (sc.factor > 0.0) {
                const double slow = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
                f = f / sc.factor * slow + f * (1.0 - slow);
            }
            for (int p = 0; p < n; p++) {
                hc[(size_t)p * half + i] = (float)(gain * std::cos(p * f));
                hs[(size_t)p * half + i] = (float)(gain * std::sin(p * f));
            }
        }
        RotTable r{dims, base, sc, nullptr, nullptr};
        TLB_TRY(upload(&r.cos_t, hc));
        TLB_TRY(upload(&r.sin_t, hs));
        lm->rots.push_back(r);
        *c = r.cos_t; *s = r.sin_t;
        return TLB_OK;
    }

    // the tensors of a layer
    tlb_status weights(Layer *L, const LayerDesc &d, int idx)
    {
        const std::string p = "l" + std::to_string(idx) + ".", q = p + "mix.";
        const MixerDesc &x = d.mix;
        const int W = lm->desc.width, H = x.heads, D = x.dim, DV = x.vdim;
        const uint64_t before = lm->weight_bytes;
        L->out_width = x.kind == MixerKind::MinGru ? x.width : H * DV;
        std::vector<Part> in;
        int n_in = 0;
        auto add = [&](const std::string &name, int n, bool bias) { in.push_back({name, n, bias}); n_in += n; return n_in - n; };
        switch (x.kind) {
        case MixerKind::Attention: {
            if (!mix_attn_supported(D, DV)) return fail(TLB_ERR_SHAPE, "layer %d: attention head sizes %d / %d (up to 256 are supported)", idx, D, DV);
            add(q + "q", H * D, x.qkv_bias); add(q + "k", x.kv_heads * D, x.qkv_bias); add(q + "v", x.kv_heads * DV, x.qkv_bias);
            const int window = std::min(x.window > 0 ? x.window : lm->cfg.max_seq, lm->cfg.max_seq);
            if (x.log_distance_bias) {
                tlb_tensor *r1, *r2;
                TLB_TRY(vec(q + "r1", &r1, H));
                TLB_TRY(vec(q + "r2", &r2, H));
                std::vector<float> a, b, t((size_t)H * window);
                TLB_TRY(host(r1, &a));
                TLB_TRY(host(r2, &b));
                for (int h = 0; h < H; h++)
                    for (int i = 0; i < window; i++) t[(size_t)h * window + i] = (float)((double)a[h] * std::log1p((double)b[h] * i));
                TLB_TRY(upload(&L->bias, t));
                L->bias_n = window;
            }
            if (x.sink) TLB_TRY(vec(q + "sink", &L->sink, H));
            break;
        }
        case MixerKind::Retention:
            if (!mix_recur_supported(D, DV)) return fail(TLB_ERR_SHAPE, "layer %d: recurrent head sizes %d / %d (up to 256 / 4096 are supported)", idx, D, DV);
            add(q + "q", H * D, false); add(q + "k", H * D, false); add(q + "v", H * DV, false); add(q + "g", H * DV, false);
            TLB_TRY(upload(&L->decay, x.decay));
            if (x.rot_dims) TLB_TRY(rotation(x.rot_dims, x.rot_base, x.rot_scaling, &L->rot_cos, &L->rot_sin));
            break;
        case MixerKind::GeneralDelta: {
            if (!mix_recur_supported(D, DV)) return fail(TLB_ERR_SHAPE, "layer %d: recurrent head sizes %d / %d (up to 256 / 4096 are supported)", idx, D, DV);
            const tlb_tensor *w1 = map_raw_bf16(m, q + "w1");
            if (!w1 || w1->rank != 2 || w1->shape[0] < 1 || w1->shape[0] > 4096) return fail(TLB_ERR_ARG, "tensor '%sw1' is missing or not a bf16 matrix", q.c_str());
            const int rank = (int)w1->shape[0], ldh = act_ld(rank);
            const_cast<LayerDesc &>(d).mix.rank = rank;
            add(q + "r", H * D, false); add(q + "k", H * D, false); add(q + "v", H * D, false); add(q + "g", H * D, false); add(q + "a", H * D, true); add(q + "w1", rank, false);
            // the second step of the decay's projection, twice side by side: its input comes as value and remainder
            const tlb_tensor *w2;
            TLB_TRY(matrix(q + "w2", &w2, H * D, rank));
            __nv_bfloat16 *dst;
            TLB_TRY(alloc(lm, &dst, (size_t)H * D * 2 * ldh));
            for (int half = 0; half < 2; half++) TLB_TRY(launch_pack_rows((const __nv_bfloat16 *)w2->data(), H * D, rank, dst, 2 * ldh, half * ldh));
            L->w2.w = dst; L->w2.n = H * D; L->w2.k = L->w2.ld = 2 * ldh;
            TLB_TRY(vec(q + "w0", &L->w0, H * D));
            TLB_TRY(vec(q + "norm", &L->onorm, H * DV));
            break;
        }
        case MixerKind::Latent:
            add(x.q_rank ? q + "dq" : q + "q", x.q_rank ? x.q_rank : H * (D + x.rot_dim), false);
            L->c_kv = add(q + "dkv", x.kv_rank + x.rot_dim, false);
            if (x.out_gate) L->c_gate = add(q + "g", H * DV, false);
            if (x.q_rank) {
                TLB_TRY(vec(q + "dq.norm", &L->qnorm, x.q_rank));
                TLB_TRY(stack(&L->uq, {{q + "uq", H * (D + x.rot_dim), false}}, x.q_rank));
            }
            TLB_TRY(vec(q + "dkv.norm", &L->cnorm, x.kv_rank));
            TLB_TRY(stack(&L->uk, {{q + "uk", H * D, false}}, x.kv_rank));
            TLB_TRY(stack(&L->uv, {{q + "uv", H * DV, false}}, x.kv_rank));
            if (!lm->cfg.f32) {
                TLB_TRY(as_f16(&L->uk16, q + "uk", H * D, x.kv_rank));
                TLB_TRY(as_f16(&L->uv16, q + "uv", H * DV, x.kv_rank));
            }
            TLB_TRY(rotation(x.rot_dims, x.rot_base, x.rot_scaling, &L->rot_cos, &L->rot_sin));
            break;
        case MixerKind::MinGru:
            add(q + "z", x.width, true); add(q + "x", x.width, true); add(q + "g", x.width, false);
            break;
        }
        if (d.resid_gate) L->c_rg1 = add(p + "rg1", W, true);
        TLB_TRY(stack(&L->in, in, W));
        TLB_TRY(stack(&L->o, {{q + "o", W, false}}, L->out_width));
        TLB_TRY(vec(p + "norm1", &L->norm1, W));
        if (d.post_norm) TLB_TRY(vec(p + "norm1b", &L->post1, W));
        if (d.layer_scale) TLB_TRY(vec(p + "ls1", &L->ls1, W));
        uint64_t idle = 0;                                   // experts a token does not read
        if (d.ffn.ff) {
            const FfnDesc &f = d.ffn;
            in.clear();
            n_in = 0;
            std::vector<Glu> pairs;
            const int act = f.act == FfnAct::SiluGlu ? GLU_SILU : GLU_GELU_TANH;
            if (f.act == FfnAct::PolyNorm) {
                add(p + "mlp.up", f.ff, false);
                TLB_TRY(vec(p + "mlp.act", &L->act, 4));
            } else if (!f.experts) {
                pairs.push_back({p + "mlp.gate", p + "mlp.up", f.ff});
            } else if (f.shared_ff) {
                pairs.push_back({p + "mlp.shared.gate", p + "mlp.shared.up", f.shared_ff});
            }
            if (d.resid_gate) L->u_rg2 = add(p + "rg2", W, true);
            if (f.experts) {
                L->route.experts = f.experts; L->route.groups = f.groups; L->route.keep = f.keep; L->route.top = f.top; L->route.scale = f.router_scale;
                if (!experts_matvec_supported(L->route, f.ff, f.shared_ff)) return fail(TLB_ERR_SHAPE, "layer %d: %d experts of %d hidden units do not fit the matvec", idx, f.top, f.ff);
                L->u_router = add(p + "mlp.router", f.experts, false);
                if (f.shared_ff) {
                    L->u_sg = add(p + "mlp.shared.sg", 1, false);
                    TLB_TRY(stack(&L->sdown, {{p + "mlp.shared.down", W, false}}, f.shared_ff));
                }
                std::vector<Glu> eu;
                std::vector<Part> ed;
                for (int e = 0; e < f.experts; e++) {
                    const std::string ep = p + "mlp.e" + std::to_string(e) + ".";
                    eu.push_back({ep + "gate", ep + "up", f.ff});
                    ed.push_back({ep + "down", W, false});
                }
                const uint64_t b0 = lm->weight_bytes;
                TLB_TRY(stack(&L->eup, {}, W, eu, act));
                TLB_TRY(stack(&L->edown, ed, f.ff));
                L->eup.n = L->eup.glu = glu_rows(f.ff); L->edown.n = W;         // rows of one expert
                idle = (lm->weight_bytes - b0) / f.experts * (f.experts - f.top);
            } else {
                TLB_TRY(stack(&L->down, {{p + "mlp.down", W, false}}, f.ff));
            }
            TLB_TRY(stack(&L->up, in, W, pairs, act));
            TLB_TRY(vec(p + "norm2", &L->norm2, W));
            if (d.post_norm) TLB_TRY(vec(p + "norm2b", &L->post2, W));
            if (d.layer_scale) TLB_TRY(vec(p + "ls2", &L->ls2, W));
        }
        L->step_bytes = lm->weight_bytes - before - idle;
        for (const DenseW *w : {&L->in, &L->o, &L->up, &L->down, &L->uq})
            if (w->w && !dense_matvec_supported(w->k)) return fail(TLB_ERR_SHAPE, "layer %d: a linear layer over %d inputs does not fit the matvec", idx, w->k);
        return TLB_OK;
    }

    // its cache or state
    tlb_status state(Layer *L, const LayerDesc &d, int idx)
    {
        const MixerDesc &x = d.mix;
        const size_t B = lm->cfg.batch, es = lm->cfg.f32 ? 4 : 2, rows = B * lm->cfg.max_seq;
        L->d = &d;
        switch (x.kind) {
        case MixerKind::Attention:
            TLB_TRY(alloc(lm, (char **)&L->kcache, rows * x.kv_heads * act_ld(x.dim) * es));
            return alloc(lm, (char **)&L->vcache, rows * x.kv_heads * act_ld(x.vdim) * es);
        case MixerKind::Latent:
            if (!latent_supported(latent_args(lm, *L, nullptr, 0, nullptr, 0), lm->cfg.f32)) return fail(TLB_ERR_SHAPE, "layer %d: latent attention over %d + %d cached values is not supported", idx, x.kv_rank, x.rot_dim);
            return alloc(lm, (char **)&L->kcache, rows * latent_ld(x.kv_rank, x.rot_dim) * es);
        case MixerKind::MinGru:
            return alloc(lm, &L->state, B * x.width);
        default:
            return alloc(lm, &L->state, B * x.heads * x.vdim * mix_recur_ld(x.dim));
        }
    }
};

MixAttn attn_args(const LayeredModel *lm, const Layer &L, const float *proj, int ldp)
{
    const MixerDesc &x = L.d->mix;
    MixAttn a = {};
    a.H = x.heads; a.KVH = x.kv_heads; a.D = x.dim; a.DV = x.vdim; a.ldk = act_ld(x.dim); a.ldv = act_ld(x.vdim);
    a.max_seq = lm->cfg.max_seq; a.window = std::min(x.window > 0 ? x.window : lm->cfg.max_seq, lm->cfg.max_seq);
    a.scale = x.scale; a.bias = L.bias; a.bias_n = L.bias_n; a.sink = L.sink ? L.sink->f32() : nullptr;
    a.kcache = L.kcache; a.vcache = L.vcache;
    a.seq_stride_k = (size_t)x.kv_heads * lm->cfg.max_seq * a.ldk; a.seq_stride_v = (size_t)x.kv_heads * lm->cfg.max_seq * a.ldv;
    a.proj = proj; a.ldp = ldp;
    return a;
}

MixRecur recur_args(const LayeredModel *lm, const Layer &L, float *proj, int ldp)
{
    const MixerDesc &x = L.d->mix;
    MixRecur r = {};
    r.H = x.heads; r.D = x.dim; r.DV = x.vdim; r.ld = mix_recur_ld(x.dim);
    r.state = L.state; r.seq_stride = (size_t)x.heads * x.vdim * r.ld;
    r.eps = lm->desc.eps; r.decay = L.decay; r.rot_cos = L.rot_cos; r.rot_sin = L.rot_sin; r.rot = x.rot_dims;
    r.norm_w = L.onorm ? L.onorm->f32() : nullptr;
    r.w2 = L.w2; r.w0 = L.w0 ? L.w0->f32() : nullptr; r.rank = x.rank;
    r.proj = proj; r.ldp = ldp;
    return r;
}

MixGru gru_args(const LayeredModel *lm, const Layer &L, const float *proj, int ldp)
{
    return MixGru{L.d->mix.width, L.state, proj, ldp};
}

// The mixer of one token per sequence: projection rows in, gated / attended rows out.
tlb_status decode_mixer(LayeredModel *lm, const Layer &L, int batch, float *proj, float *q, void *qa, float *latent_partial, const int *pos, const int *rope_pos, void *out,
                        int ldo, bool out_f32, bool pdl)
{
    switch (L.d->mix.kind) {
    case MixerKind::Attention: {
        MixAttnDecode j = {};
        j.a = attn_args(lm, L, proj, lm->ldp);
        j.batch = batch; j.pos = pos; j.partial = lm->partial; j.counters = lm->counters; j.out = out; j.ldo = ldo;
        j.out_f32 = out_f32; j.cache_f32 = lm->cfg.f32; j.pdl = pdl;
        return launch_mix_attn_decode(j);
    }
    case MixerKind::Latent: {
        MixLatentRows j = {};
        j.m = latent_args(lm, L, proj, lm->ldp, q, lm->ldq);
        j.rows = batch; j.seq_step = 1; j.pos = pos; j.rope_pos = rope_pos; j.qa = qa; j.partial = latent_partial; j.out = out; j.ldo = ldo;
        j.f32 = lm->cfg.f32; j.out_f32 = out_f32; j.pdl = pdl;
        return launch_latent_rows(j);
    }
    case MixerKind::MinGru:
        return launch_gru_rows(gru_args(lm, L, proj, lm->ldp), batch, pos, out, ldo, out_f32, pdl);
    default: {
        MixRecurDecode j = {};
        j.m = recur_args(lm, L, proj, lm->ldp);
        j.batch = batch; j.pos = pos; j.rope_pos = rope_pos; j.out = out; j.ldo = ldo; j.out_f32 = out_f32; j.pdl = pdl;
        return L.d->mix.kind == MixerKind::Retention ? launch_retention_decode(j) : launch_delta_decode(j);
    }
    }
}

// Storage of one pass, given back at its end.
struct Rows {
    std::vector<Storage *> all;
    tlb_status operator()(void **p, size_t bytes)
    {
        Storage *s = storage_alloc(bytes);
        if (!s) return TLB_ERR_ALLOC;
        all.push_back(s);
        *p = s->ptr;
        return TLB_OK;
    }
    template <typename T> tlb_status get(T **p, size_t bytes) { return (*this)((void **)p, bytes); }
    ~Rows() { for (Storage *s : all) storage_release(s); }
};

// Work rows for T rows, from get(pointer, bytes); x apart.  absorbed: rows of latent attention queries stay in the latent space.
template <typename Get>
tlb_status row_bufs(const LayeredModel *lm, int T, bool absorbed, RowBufs *b, Get get)
{
    const size_t es = lm->cfg.f32 ? 4 : 2, W = lm->desc.width;
    size_t n_dly = 0, n_th = 0, n_look = 0, n_y = 0, top = 0, experts = 0, ld_ff = 0, ld_hid = 0, tiles = 0, shared = 0, n_qa = 0, n_part = 0;
    for (const Layer &L : lm->layers) {
        if (L.d->mix.kind == MixerKind::GeneralDelta) { n_dly = std::max(n_dly, (size_t)L.w2.n); n_th = std::max(n_th, (size_t)L.w2.k); n_look = std::max(n_look, (size_t)L.d->mix.heads); }
        if (L.d->post_norm) n_y = W;
        if (L.eup.w) {
            top = std::max(top, (size_t)L.route.top); experts = std::max(experts, (size_t)L.route.experts);
            ld_ff = std::max(ld_ff, (size_t)act_ld(L.edown.k));
            tiles = std::max(tiles, (size_t)moe_max_tiles(L.route, T, lm->cfg.f32));
            if (L.sdown.w) shared = W;
        }
        if (L.up.glu) ld_hid = std::max(ld_hid, (size_t)act_ld(L.up.glu / 2));
        if (absorbed && L.d->mix.kind == MixerKind::Latent) {
            const MixLatent m = latent_args(lm, L, nullptr, 0, nullptr, 0);
            n_qa = std::max(n_qa, (size_t)m.H * m.ld); n_part = std::max(n_part, latent_partial_floats(m, T));
        }
    }
    const size_t t = T;
    auto want = [&](auto **p, size_t bytes) { return bytes ? get((void **)p, bytes) : TLB_OK; };
    TLB_TRY(want(&b->proj, t * lm->ldp * 4));
    TLB_TRY(want(&b->u, t * lm->ldu * 4));
    TLB_TRY(want(&b->o, t * lm->ldm * 4));
    TLB_TRY(want(&b->act, t * lm->lda * es));
    TLB_TRY(want(&b->y, t * n_y * 4));
    TLB_TRY(want(&b->q, t * lm->ldq * 4));
    TLB_TRY(want(&b->dly, t * n_dly * 4));
    TLB_TRY(want(&b->th, t * n_th * es));
    TLB_TRY(want(&b->look, (size_t)scan_look_ld(T) * n_look * sizeof(float2)));
    TLB_TRY(want(&b->plan.sel, t * top * 4));
    TLB_TRY(want(&b->plan.place, t * top * 4));
    TLB_TRY(want(&b->plan.weight, t * top * 4));
    TLB_TRY(want(&b->plan.count, 2 * experts * 4));
    TLB_TRY(want(&b->plan.tiles, tiles * sizeof(int4)));
    TLB_TRY(want(&b->hid, t * ld_hid * es));
    TLB_TRY(want(&b->hp, t * top * ld_ff * es));
    TLB_TRY(want(&b->yp, t * top * W * 4));
    TLB_TRY(want(&b->xp, t * top * act_ld((int)W) * es));
    TLB_TRY(want(&b->ysh, t * shared * 4));
    TLB_TRY(want(&b->qa, t * n_qa * es));
    return want(&b->partial, n_part * 4);
}

tlb_status rows_gemm(const LayeredModel *lm, const DenseW &w, const void *x, int ldx, int T, float *out, int ldo, const tlb_tensor *scale, float softcap = 0.f, void *hid = nullptr)
{
    DenseGemmJob j;
    j.act_out = hid; j.ld_act = act_ld(w.glu / 2);
    j.w = w; j.x = x; j.ldx = ldx; j.T = T; j.out = out; j.ldo = ldo; j.resid_scale = scale ? scale->f32() : nullptr; j.softcap = softcap;
    return launch_dense_gemm(j, lm->cfg.f32);
}

// rows of the residual through a norm of the width, in the activation type
tlb_status rows_norm(const LayeredModel *lm, const float *x, int T, const tlb_tensor *w, void *out)
{
    const ModelDesc &d = lm->desc;
    const int ld = act_ld(d.width);
    if (d.norm_groups == 1) return launch_norm_rows(x, T, d.width, d.width, w->f32(), d.norm_offset, d.eps, out, ld, lm->cfg.f32);
    ResidNormJob j;
    j.x = const_cast<float *>(x); j.T = T; j.width = d.width; j.groups = d.norm_groups; j.offset = d.norm_offset; j.eps = d.eps; j.norm_w = w->f32(); j.out = out; j.ldo = ld;
    return launch_resid_norm_rows(j, lm->cfg.f32);
}

// The mixer over rows: b.proj -> b.act.
tlb_status rows_mixer(LayeredModel *lm, const Layer &L, RowBufs &b, const RowCtx &c, int lda)
{
    const bool f32 = lm->cfg.f32;
    const MixerDesc &x = L.d->mix;
    if (x.q_rank) {
        TLB_TRY(launch_norm_rows(b.proj, c.T, x.q_rank, lm->ldp, L.qnorm->f32(), 0.f, lm->desc.eps, b.act, act_ld(x.q_rank), f32));
        TLB_TRY(rows_gemm(lm, L.uq, b.act, act_ld(x.q_rank), c.T, b.q, lm->ldq, nullptr));
    }
    if (c.pos) return decode_mixer(lm, L, c.T, b.proj, b.q, b.qa, b.partial, c.pos, c.rope, b.act, lda, f32, false);
    switch (x.kind) {
    case MixerKind::Attention:
        return launch_mix_attn_prefill(attn_args(lm, L, b.proj, lm->ldp), c.seq, c.T, c.pos0, b.act, lda, f32);
    case MixerKind::Retention:
        return launch_retention_prefill(recur_args(lm, L, b.proj, lm->ldp), c.seq, c.T, c.pos0, c.rope0, c.rope_step, b.o, b.act, lda, f32);
    case MixerKind::GeneralDelta:
        TLB_TRY(launch_tanh_split(b.proj + 5 * (size_t)L.w2.n, c.T, x.rank, lm->ldp, b.th, L.w2.k / 2, f32));
        TLB_TRY(rows_gemm(lm, L.w2, b.th, L.w2.k, c.T, b.dly, L.w2.n, nullptr));
        return launch_delta_prefill(recur_args(lm, L, b.proj, lm->ldp), c.seq, c.T, c.pos0, b.dly, b.look, b.o, b.act, lda, f32);
    case MixerKind::Latent: {
        const MixLatent m = latent_args(lm, L, b.proj, lm->ldp, b.q, lm->ldq);
        if (latent_expands(m, c.T)) return launch_latent_prompt(m, c.seq, c.T, c.pos0, c.rope0, c.rope_step, b.act, lda, f32);
        MixLatentRows j = {};
        j.m = m; j.rows = c.T; j.seq0 = c.seq; j.pos0 = c.pos0; j.rope0 = c.rope0; j.rope_step = c.rope_step; j.qa = b.qa; j.partial = b.partial; j.out = b.act; j.ldo = lda;
        j.f32 = j.out_f32 = f32;
        return launch_latent_rows(j);
    }
    case MixerKind::MinGru:
        return launch_gru_prefill(gru_args(lm, L, b.proj, lm->ldp), c.seq, c.T, c.pos0, b.act, lda, f32);
    }
    return TLB_OK;
}

// The mixture of experts over rows: normed rows in b.act, of the first projection the shared activations in b.hid, the rest in b.u.
tlb_status rows_experts(LayeredModel *lm, const Layer &L, RowBufs &b, int T, MoeRows *out)
{
    const bool f32 = lm->cfg.f32;
    const int W = lm->desc.width, ff = L.edown.k, ldw = act_ld(W), ldf = act_ld(ff), P = T * L.route.top;
    TLB_TRY(launch_moe_plan(L.route, b.u + L.u_router, lm->ldu, T, b.plan, f32));
    TLB_TRY(launch_moe_gather(L.route, b.plan, b.act, T, ldw, b.xp, f32));
    DenseGemmJob j;
    j.tiles = b.plan.tiles; j.n_tiles = moe_max_tiles(L.route, T, f32); j.tile_rows = moe_tile_rows(L.route, T, f32); j.n_weights = L.route.experts; j.T = P;
    j.w = L.eup; j.x = b.xp; j.ldx = ldw; j.act_out = b.hp; j.ld_act = ldf;
    TLB_TRY(launch_dense_gemm(j, f32));
    j.w = L.edown; j.x = b.hp; j.ldx = ldf; j.out = b.yp; j.ldo = W;
    TLB_TRY(launch_dense_gemm(j, f32));
    out->top = L.route.top; out->slot = b.plan.place; out->weight = b.plan.weight; out->part = b.yp;
    if (L.sdown.w) {
        TLB_TRY(rows_gemm(lm, L.sdown, b.hid, act_ld(L.sdown.k), T, b.ysh, W, nullptr));
        out->shared = b.ysh; out->shared_gate = b.u + L.u_sg; out->ld_shared_gate = lm->ldu;
    }
    return TLB_OK;
}

// All layers over rows of the residual in b.x.
tlb_status run_rows(LayeredModel *lm, RowBufs &b, const RowCtx &c)
{
    const ModelDesc &md = lm->desc;
    const int W = md.width, T = c.T, ldw = act_ld(W);
    const bool f32 = lm->cfg.f32;
    // what a sublayer left joins the residual, and the next norm (null: none) follows
    auto join = [&](const Layer &L, const MoeRows *moe, const float *gate, int ldg, const tlb_tensor *post, const tlb_tensor *next) -> tlb_status {
        if (!L.d->post_norm) return next ? rows_norm(lm, b.x, T, next, b.act) : TLB_OK;          // the projection has added it
        ResidNormJob j;
        j.x = b.x; j.T = T; j.width = W; j.groups = md.norm_groups; j.offset = md.norm_offset; j.eps = md.eps;
        j.y = moe ? nullptr : b.y; j.moe = moe; j.gate = gate; j.ld_gate = ldg; j.post_w = post->f32();
        j.norm_w = next ? next->f32() : nullptr; j.out = b.act; j.ldo = ldw;
        return launch_resid_norm_rows(j, f32);
    };
    TLB_TRY(rows_norm(lm, b.x, T, lm->layers[0].norm1, b.act));
    for (size_t i = 0; i < lm->layers.size(); i++) {
        const Layer &L = lm->layers[i];
        const bool post = L.d->post_norm;
        const tlb_tensor *next = i + 1 < lm->layers.size() ? lm->layers[i + 1].norm1 : nullptr;
        const int lda = act_ld(L.out_width);
        TLB_TRY(rows_gemm(lm, L.in, b.act, ldw, T, b.proj, lm->ldp, nullptr));
        TLB_TRY(rows_mixer(lm, L, b, c, lda));
        TLB_TRY(rows_gemm(lm, L.o, b.act, lda, T, post ? b.y : b.x, W, L.ls1));
        TLB_TRY(join(L, nullptr, L.c_rg1 >= 0 ? b.proj + L.c_rg1 : nullptr, lm->ldp, L.post1, L.up.w ? L.norm2 : next));
        if (!L.up.w) continue;
        TLB_TRY(rows_gemm(lm, L.up, b.act, ldw, T, b.u, lm->ldu, nullptr, 0.f, b.hid));
        MoeRows moe;
        if (L.eup.w) {
            TLB_TRY(rows_experts(lm, L, b, T, &moe));
        } else {
            const int ldf = act_ld(L.down.k);
            if (L.act) TLB_TRY(launch_poly_rows(b.u, T, L.down.k, lm->ldu, L.act->f32(), md.eps, b.act, ldf, f32));
            TLB_TRY(rows_gemm(lm, L.down, L.act ? b.act : b.hid, ldf, T, post ? b.y : b.x, W, L.ls2));
        }
        TLB_TRY(join(L, L.eup.w ? &moe : nullptr, L.u_rg2 >= 0 ? b.u + L.u_rg2 : nullptr, lm->ldu, L.post2, next));
    }
    return TLB_OK;
}

// The chain of one token: the residual and what the last sublayer left beside it.
struct Chain {
    LayeredModel *lm;
    const int *token;
    float *buf[2];                     // residual; it moves to the other one whenever a launch's prologue adds to it
    int cur = 0;
    bool first = true;
    const float *gate = nullptr;
    const tlb_tensor *post = nullptr;  // pending: lm->y waits to be gated, normed and added

    // norm -> linear layer, the pending addition in front
    tlb_status front(const DenseW &w, const tlb_tensor *norm, float *out, float *h_out = nullptr, float softcap = 0.f)
    {
        const ModelDesc &d = lm->desc;
        DenseMatvecJob j;
        j.act_out = lm->hid;
        j.w = w; j.norm_w = norm->f32(); j.norm_offset = d.norm_offset; j.eps = d.eps; j.groups = d.norm_groups; j.out = out; j.h_out = h_out; j.softcap = softcap;
        j.pro = d.norm_groups > 1 || post || h_out ? DPRO_GNORM : DPRO_NORM;
        j.x = buf[cur];
        if (first) { j.emb = lm->embed; j.token = token; j.x_out = buf[cur]; }
        if (post) { j.y = lm->y; j.y_gate = gate; j.post_w = post->f32(); cur ^= 1; j.x_out = buf[cur]; }
        first = false;
        post = nullptr;
        return launch_dense_matvec(j);
    }
    // the last linear layer of a sublayer
    tlb_status back(DenseMatvecJob &j, const Layer &L, const tlb_tensor *scale, const tlb_tensor *post_norm, const float *resid_gate)
    {
        if (L.d->post_norm) { j.out = lm->y; post = post_norm; gate = resid_gate; }
        else { j.out = buf[cur]; j.resid_scale = scale->f32(); }
        return launch_dense_matvec(j);
    }
};

}  // namespace

void layered_destroy(LayeredModel *lm)
{
    if (!lm) return;
    for (tlb_tensor *t : lm->held) tlb_tensor_release(t);
    for (Storage *s : lm->stores) storage_release(s);
    delete lm;
}

tlb_status layered_create(LayeredModel **out, const ModelDesc &desc, tlb_map *m, const LayeredCfg &cfg)
{
    *out = nullptr;
    LayeredModel *lm = new LayeredModel();
    lm->desc = desc;
    lm->cfg = cfg;
    Loader ld{lm, m};
    const int W = desc.width, B = cfg.batch;
    auto build = [&]() -> tlb_status {
        DenseW e;
        TLB_TRY(ld.stack(&e, {{"embed", desc.vocab, false}}, W));
        lm->embed = e.w; lm->embed_ld = e.ld;
        lm->layers.resize(desc.layers.size());
        for (size_t i = 0; i < desc.layers.size(); i++)
            if (lm->desc.layers[i].weights_of < 0) TLB_TRY(ld.weights(&lm->layers[i], lm->desc.layers[i], (int)i));
        for (size_t i = 0; i < desc.layers.size(); i++) {
            const int of = lm->desc.layers[i].weights_of;
            if (of >= 0) {
                lm->layers[i] = lm->layers[of];          // the tensors; the cache or state is its own
                lm->desc.layers[i].mix.rank = lm->desc.layers[of].mix.rank;
            }
        }
        for (size_t i = 0; i < desc.layers.size(); i++) { lm->layers[i].d = &lm->desc.layers[i]; TLB_TRY(ld.state(&lm->layers[i], lm->desc.layers[i], (int)i)); }
        TLB_TRY(ld.stack(&lm->head, {{"head", desc.vocab, false}}, W));
        TLB_TRY(ld.vec("final.norm", &lm->final_norm, W));
        size_t part = 1, lpart = 0, qa = 0, hid = 0, ex = 0, top = 0, attn_part = 0;
        int kvh = 1;
        lm->ldp = lm->ldm = lm->ldu = 8;
        lm->lda = act_ld(W);
        for (const Layer &L : lm->layers) {
            const MixerDesc &x = L.d->mix;
            lm->ldp = std::max(lm->ldp, act_ld(L.in.n));
            lm->ldm = std::max(lm->ldm, act_ld(L.out_width));
            lm->ldu = std::max(lm->ldu, act_ld(L.up.n - L.up.glu));
            for (int n : {L.out_width, L.down.k, L.sdown.k, x.q_rank}) lm->lda = std::max(lm->lda, act_ld(n));
            if (x.kind == MixerKind::Attention) {
                attn_part = std::max(attn_part, mix_attn_decode_partial_floats(attn_args(lm, L, nullptr, 0), B));
                kvh = std::max(kvh, x.kv_heads);
            } else if (x.kind == MixerKind::Latent) {
                const MixLatent m = latent_args(lm, L, nullptr, 0, nullptr, 0);
                lpart = std::max(lpart, latent_partial_floats(m, 1));
                qa = std::max(qa, (size_t)m.H * m.ld);
                if (x.q_rank) lm->ldq = std::max(lm->ldq, act_ld(L.uq.n));
            }
            hid = std::max(hid, (size_t)L.up.glu / 2);
            if (L.eup.w) { ex = std::max(ex, (size_t)L.route.top * L.eup.n / 2); top = std::max(top, (size_t)L.route.top); }
        }
        part = std::max(part, std::max(attn_part, lpart));
        for (float *&p : lm->proj) TLB_TRY(alloc(lm, &p, lm->ldp));
        TLB_TRY(alloc(lm, &lm->mix, lm->ldm));
        TLB_TRY(alloc(lm, &lm->up, lm->ldu));
        TLB_TRY(alloc(lm, &lm->partial, part));
        TLB_TRY(alloc(lm, &lm->counters, (size_t)B * kvh));
        for (float **p : {&lm->x2, &lm->y, &lm->h}) TLB_TRY(alloc(lm, p, W));
        if (lm->ldq) TLB_TRY(alloc(lm, &lm->q, lm->ldq));
        if (hid) TLB_TRY(alloc(lm, &lm->hid, hid));
        if (qa) TLB_TRY(alloc(lm, (char **)&lm->qa, qa * (cfg.f32 ? 4 : 2)));
        if (top) { TLB_TRY(alloc(lm, &lm->ex, ex)); TLB_TRY(alloc(lm, &lm->weight, top)); TLB_TRY(alloc(lm, &lm->sel, top)); }
        if (B > 1) TLB_TRY(row_bufs(lm, B, true, &lm->batch_rows, [&](void **p, size_t bytes) { return alloc(lm, (char **)p, bytes); }));
        return tlb_sync();
    };
    tlb_status st = build();
    if (st != TLB_OK) { layered_destroy(lm); return st; }
    *out = lm;
    return TLB_OK;
}

tlb_status layered_step(LayeredModel *lm, const int *token, const int *pos, const int *rope_pos, float *x, float *logits)
{
    const float eps = lm->desc.eps;
    int moves = 0;                      // residual additions made in a prologue: the last one must leave the residual in x
    for (const Layer &L : lm->layers)
        if (L.d->post_norm) moves += L.up.w ? 2 : 1;
    Chain c;
    c.lm = lm; c.token = token; c.buf[0] = x; c.buf[1] = lm->x2; c.cur = moves & 1;
    int turn = 0;
    for (const Layer &L : lm->layers) {
        const MixerDesc &mx = L.d->mix;
        float *proj = lm->proj[turn ^= 1];
        TLB_TRY(c.front(L.in, L.norm1, proj));
        if (mx.q_rank) {
            DenseMatvecJob j;
            j.w = L.uq; j.pro = DPRO_NORM; j.x = proj; j.norm_w = L.qnorm->f32(); j.eps = eps; j.out = lm->q;
            TLB_TRY(launch_dense_matvec(j));
        }
        TLB_TRY(decode_mixer(lm, L, 1, proj, lm->q, lm->qa, lm->partial, pos, rope_pos, lm->mix, lm->ldm, true, true));
        DenseMatvecJob j;
        j.w = L.o; j.x = lm->mix;
        TLB_TRY(c.back(j, L, L.ls1, L.post1, L.c_rg1 >= 0 ? proj + L.c_rg1 : nullptr));
        if (!L.up.w) continue;
        TLB_TRY(c.front(L.up, L.norm2, lm->up, L.eup.w ? lm->h : nullptr));
        j = DenseMatvecJob();
        if (L.eup.w) {
            j.w = L.eup; j.pro = DPRO_EXPERT; j.x = lm->h; j.route = L.route; j.logits = lm->up + L.u_router; j.sel = lm->sel; j.weight = lm->weight; j.act_out = lm->ex;
            TLB_TRY(launch_dense_matvec(j));
            j.w = L.edown; j.pro = DPRO_EXPERTS; j.x = lm->ex; j.ldx = L.eup.n / 2;
            if (L.sdown.w) { j.shared = L.sdown; j.shared_x = lm->hid; j.shared_gate = lm->up + L.u_sg; }
        } else {
            j.w = L.down; j.x = L.act ? lm->up : lm->hid; j.eps = eps;
            if (L.act) { j.pro = DPRO_POLY; j.poly = L.act->f32(); }
        }
        TLB_TRY(c.back(j, L, L.ls2, L.post2, L.u_rg2 >= 0 ? lm->up + L.u_rg2 : nullptr));
    }
    return c.front(lm->head, lm->final_norm, logits, nullptr, lm->desc.logit_softcap);
}

tlb_status layered_step_batch(LayeredModel *lm, const int *tokens, const int *pos, const int *rope_pos, int batch, float *x, float *logits)
{
    TLB_TRY(launch_embed_bf16(tokens, lm->embed, lm->desc.width, lm->embed_ld, x, batch));
    RowBufs b = lm->batch_rows;
    b.x = x;
    RowCtx c;
    c.T = batch; c.pos = pos; c.rope = rope_pos;
    TLB_TRY(run_rows(lm, b, c));
    return layered_head(lm, x, batch, logits);
}

tlb_status layered_prefill(LayeredModel *lm, int seq, const int32_t *tokens, int T, int pos0, int rope0, int rope_step, const int32_t *want,
                           int n_want, float *rows_out)
{
    const int W = lm->desc.width;
    Rows ws;
    RowBufs b;
    int *ids;
    bool absorbed = false;
    for (const Layer &L : lm->layers)
        absorbed |= L.d->mix.kind == MixerKind::Latent && !latent_expands(latent_args(lm, L, nullptr, 0, nullptr, 0), T);
    TLB_TRY(ws.get(&ids, ((size_t)T + std::max(n_want, 1)) * sizeof(int)));
    TLB_TRY(ws.get(&b.x, (size_t)T * W * 4));
    TLB_TRY(row_bufs(lm, T, absorbed, &b, [&](void **p, size_t bytes) { return ws(p, bytes); }));
    // pageable sources: staged before the calls return
    TLB_CUDA(cudaMemcpyAsync(ids, tokens, (size_t)T * sizeof(int), cudaMemcpyHostToDevice, ctx()->stream));
    if (n_want) TLB_CUDA(cudaMemcpyAsync(ids + T, want, (size_t)n_want * sizeof(int), cudaMemcpyHostToDevice, ctx()->stream));
    TLB_TRY(launch_embed_bf16(ids, lm->embed, W, lm->embed_ld, b.x, T));
    RowCtx c;
    c.T = T; c.seq = seq; c.pos0 = pos0; c.rope0 = rope0; c.rope_step = rope_step;
    TLB_TRY(run_rows(lm, b, c));
    if (n_want) TLB_TRY(launch_gather_rows(b.x, W, ids + T, n_want, rows_out));
    return TLB_OK;
}

tlb_status layered_head(LayeredModel *lm, const float *rows, int n, float *logits)
{
    const int W = lm->desc.width, V = lm->desc.vocab;
    if (n == 1) {
        Chain c;
        c.lm = lm; c.token = nullptr; c.first = false; c.buf[0] = c.buf[1] = const_cast<float *>(rows);
        return c.front(lm->head, lm->final_norm, logits, nullptr, lm->desc.logit_softcap);
    }
    Rows ws;
    void *act;
    TLB_TRY(ws.get(&act, (size_t)n * act_ld(W) * (lm->cfg.f32 ? 4 : 2)));
    TLB_TRY(rows_norm(lm, rows, n, lm->final_norm, act));
    return rows_gemm(lm, lm->head, act, act_ld(W), n, logits, V, nullptr, lm->desc.logit_softcap);
}

uint64_t layered_weight_bytes(const LayeredModel *lm)
{
    uint64_t b = ((uint64_t)lm->desc.vocab + 1) * lm->desc.width * 2 + (uint64_t)lm->desc.width * 4;      // head, one embedding row, last norm
    for (const Layer &L : lm->layers) b += L.step_bytes;
    return b;
}

uint64_t layered_state_bytes(const LayeredModel *lm, int ctx_len)
{
    uint64_t b = 0;
    for (const Layer &L : lm->layers) {
        const MixerDesc &x = L.d->mix;
        const uint64_t seen = std::min(ctx_len, x.window > 0 ? x.window : ctx_len), es = lm->cfg.f32 ? 4 : 2;
        switch (x.kind) {
        case MixerKind::Attention: b += seen * x.kv_heads * (x.dim + x.vdim) * es; break;
        case MixerKind::Latent: b += seen * (x.kv_rank + x.rot_dim) * es; break;
        case MixerKind::MinGru: b += 2ull * x.width * 4; break;                  // read and written
        default: b += 2ull * x.heads * x.vdim * mix_recur_ld(x.dim) * 4;
        }
    }
    return b;
}

int layered_kernels_per_step(const LayeredModel *lm)
{
    int n = 1;
    for (const Layer &L : lm->layers) {
        const MixerDesc &x = L.d->mix;
        n += x.kind == MixerKind::Latent ? (x.q_rank ? 6 : 5) : 3;
        n += !L.up.w ? 0 : (L.eup.w ? 3 : 2);
    }
    return n;
}

}  // namespace tlb
