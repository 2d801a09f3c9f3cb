// A decoder described as a list of layers (model_desc.h), each with one of several mixers and an optional feed-forward: weights
// stacked per launch, caches and recurrent state per sequence, and the three ways a session runs it.
//   one token      norm -> stacked input projections | mixer | output projection -> residual | norm -> up | activation -> down
//                  -> residual: five launches a layer (three without a feed-forward), chained with programmatic dependent launch
//   one token of every sequence of a batch, and T tokens of one sequence: the same steps over rows, linear layers as GEMMs
// The residual, norms, scores, recurrences and everything that enters them stay in 32-bit floats.
#include "model_desc.h"

#include <algorithm>
#include <cmath>

#include "layered_kernels.h"

namespace tlb {

namespace {

struct Layer {
    const LayerDesc *d = nullptr;
    DenseW in, o, up, down, w2;
    tlb_tensor *norm1 = nullptr, *norm2 = nullptr, *ls1 = nullptr, *ls2 = nullptr, *act = nullptr;
    tlb_tensor *sink = nullptr, *onorm = nullptr, *w0 = nullptr;
    float *bias = nullptr;                 // by distance, [heads][bias_n]
    int bias_n = 0;
    float *decay = nullptr, *rot_cos = nullptr, *rot_sin = nullptr;
    void *kcache = nullptr, *vcache = nullptr;
    float *state = nullptr;
    int out_width = 0;                     // columns the output projection reads
};

struct RotTable { int dims; double base; float *cos_t, *sin_t; };

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
    // rows of the batch: projections, mixer output, up projection (f32); activation rows of the batch path
    float *proj = nullptr, *mix = nullptr, *up = nullptr, *partial = nullptr;
    void *act = nullptr;
    int *counters = nullptr;
    int ldp = 0, ldm = 0, ldu = 0, lda = 0;
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
    tlb_status stack(DenseW *w, const std::vector<Part> &parts, int k)
    {
        int n = 0;
        bool any_bias = false;
        for (const Part &p : parts) { n += p.n; any_bias |= p.bias; }
        w->n = n; w->k = k; w->ld = act_ld(k);
        if (parts.size() == 1 && w->ld == k) {
            const tlb_tensor *t;
            TLB_TRY(matrix(parts[0].name, &t, n, k));
            tlb_tensor_retain(const_cast<tlb_tensor *>(t));
            lm->held.push_back(const_cast<tlb_tensor *>(t));
            w->w = (const __nv_bfloat16 *)t->data();
        } else {
            __nv_bfloat16 *dst;
            TLB_TRY(alloc(lm, &dst, (size_t)n * w->ld, w->ld != k));
            int at = 0;
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
            int at = 0;
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

    // cos / sin of p * base^(-2 i / dims) for every position, angles in double
    tlb_status rotation(int dims, double base, float **c, float **s)
    {
        for (const RotTable &r : lm->rots)
            if (r.dims == dims && r.base == base) { *c = r.cos_t; *s = r.sin_t; return TLB_OK; }
        const int half = dims / 2, n = lm->cfg.max_seq;
        std::vector<float> hc((size_t)n * half), hs((size_t)n * half);
        for (int i = 0; i < half; i++) {
            const double f = std::pow(base, -2.0 * i / dims);
            for (int p = 0; p < n; p++) {
                hc[(size_t)p * half + i] = (float)std::cos(p * f);
                hs[(size_t)p * half + i] = (float)std::sin(p * f);
            }
        }
        RotTable r{dims, base, nullptr, nullptr};
        TLB_TRY(upload(&r.cos_t, hc));
        TLB_TRY(upload(&r.sin_t, hs));
        lm->rots.push_back(r);
        *c = r.cos_t; *s = r.sin_t;
        return TLB_OK;
    }

    tlb_status layer(Layer *L, const LayerDesc &d, int idx)
    {
        const std::string p = "l" + std::to_string(idx) + ".", q = p + "mix.";
        const MixerDesc &x = d.mix;
        const int W = lm->desc.width, H = x.heads, D = x.dim, DV = x.vdim, B = lm->cfg.batch;
        L->d = &d;
        L->out_width = H * DV;
        if (x.kind == MixerKind::Attention) {
            if (!mix_attn_supported(D, DV)) return fail(TLB_ERR_SHAPE, "layer %d: attention head sizes %d / %d (up to 256 are supported)", idx, D, DV);
            TLB_TRY(stack(&L->in, {{q + "q", H * D, x.qkv_bias}, {q + "k", x.kv_heads * D, x.qkv_bias}, {q + "v", x.kv_heads * DV, x.qkv_bias}}, W));
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
            const size_t es = lm->cfg.f32 ? 4 : 2, rows = (size_t)B * x.kv_heads * lm->cfg.max_seq;
            TLB_TRY(alloc(lm, (char **)&L->kcache, rows * act_ld(D) * es));
            TLB_TRY(alloc(lm, (char **)&L->vcache, rows * act_ld(DV) * es));
        } else {
            if (!mix_recur_supported(D, DV)) return fail(TLB_ERR_SHAPE, "layer %d: recurrent head sizes %d / %d (up to 256 / 4096 are supported)", idx, D, DV);
            if (x.kind == MixerKind::Retention) {
                TLB_TRY(stack(&L->in, {{q + "q", H * D, false}, {q + "k", H * D, false}, {q + "v", H * DV, false}, {q + "g", H * DV, false}}, W));
                TLB_TRY(upload(&L->decay, x.decay));
                if (x.rot_dims) TLB_TRY(rotation(x.rot_dims, x.rot_base, &L->rot_cos, &L->rot_sin));
            } else {
                const tlb_tensor *w1 = map_raw_bf16(m, q + "w1");
                if (!w1 || w1->rank != 2 || w1->shape[0] < 1 || w1->shape[0] > 4096) return fail(TLB_ERR_ARG, "tensor '%sw1' is missing or not a bf16 matrix", q.c_str());
                const int rank = (int)w1->shape[0], ldh = act_ld(rank);
                const_cast<LayerDesc &>(d).mix.rank = rank;
                TLB_TRY(stack(&L->in, {{q + "r", H * D, false}, {q + "k", H * D, false}, {q + "v", H * D, false}, {q + "g", H * D, false}, {q + "a", H * D, true}, {q + "w1", rank, false}}, W));
                // the second step of the decay's projection, twice side by side: its input comes as value and remainder
                const tlb_tensor *w2;
                TLB_TRY(matrix(q + "w2", &w2, H * D, rank));
                __nv_bfloat16 *dst;
                TLB_TRY(alloc(lm, &dst, (size_t)H * D * 2 * ldh));
                for (int half = 0; half < 2; half++) TLB_TRY(launch_pack_rows((const __nv_bfloat16 *)w2->data(), H * D, rank, dst, 2 * ldh, half * ldh));
                L->w2.w = dst; L->w2.n = H * D; L->w2.k = L->w2.ld = 2 * ldh;
                TLB_TRY(vec(q + "w0", &L->w0, H * D));
                TLB_TRY(vec(q + "norm", &L->onorm, H * DV));
            }
            TLB_TRY(alloc(lm, &L->state, (size_t)B * H * DV * mix_recur_ld(D)));
        }
        TLB_TRY(stack(&L->o, {{q + "o", W, false}}, H * DV));
        TLB_TRY(vec(p + "norm1", &L->norm1, W));
        if (d.layer_scale) TLB_TRY(vec(p + "ls1", &L->ls1, W));
        if (d.ffn.ff) {
            TLB_TRY(stack(&L->up, {{p + "mlp.up", d.ffn.ff, false}}, W));
            TLB_TRY(stack(&L->down, {{p + "mlp.down", W, false}}, d.ffn.ff));
            TLB_TRY(vec(p + "mlp.act", &L->act, 4));
            TLB_TRY(vec(p + "norm2", &L->norm2, W));
            if (d.layer_scale) TLB_TRY(vec(p + "ls2", &L->ls2, W));
        }
        for (const DenseW *w : {&L->in, &L->o, &L->up, &L->down})
            if (w->w && !dense_matvec_supported(w->k)) return fail(TLB_ERR_SHAPE, "layer %d: a linear layer over %d inputs does not fit the matvec", idx, w->k);
        return TLB_OK;
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

// The mixer of one token per sequence: projection rows in lm->proj, gated / attended rows out.
tlb_status decode_mixer(LayeredModel *lm, const Layer &L, int batch, const int *pos, const int *rope_pos, void *out, int ldo, bool out_f32, bool pdl)
{
    if (L.d->mix.kind == MixerKind::Attention) {
        MixAttnDecode j = {};
        j.a = attn_args(lm, L, lm->proj, lm->ldp);
        j.batch = batch; j.pos = pos; j.partial = lm->partial; j.counters = lm->counters; j.out = out; j.ldo = ldo;
        j.out_f32 = out_f32; j.cache_f32 = lm->cfg.f32; j.pdl = pdl;
        return launch_mix_attn_decode(j);
    }
    MixRecurDecode j = {};
    j.m = recur_args(lm, L, lm->proj, lm->ldp);
    j.batch = batch; j.pos = pos; j.rope_pos = rope_pos; j.out = out; j.ldo = ldo; j.out_f32 = out_f32; j.pdl = pdl;
    return L.d->mix.kind == MixerKind::Retention ? launch_retention_decode(j) : launch_delta_decode(j);
}

// Work rows of a pass over `T` rows, in the activation type.
struct Rows {
    std::vector<Storage *> all;
    template <typename T> tlb_status get(T **p, size_t bytes)
    {
        Storage *s = storage_alloc(bytes);
        if (!s) return TLB_ERR_ALLOC;
        all.push_back(s);
        *p = (T *)s->ptr;
        return TLB_OK;
    }
    ~Rows() { for (Storage *s : all) storage_release(s); }
};

tlb_status rows_gemm(const LayeredModel *lm, const DenseW &w, const void *x, int ldx, int T, float *out, int ldo, const tlb_tensor *scale)
{
    DenseGemmJob j;
    j.w = w; j.x = x; j.ldx = ldx; j.T = T; j.out = out; j.ldo = ldo; j.resid_scale = scale ? scale->f32() : nullptr;
    return launch_dense_gemm(j, lm->cfg.f32);
}

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
        for (size_t i = 0; i < desc.layers.size(); i++) TLB_TRY(ld.layer(&lm->layers[i], lm->desc.layers[i], (int)i));
        TLB_TRY(ld.stack(&lm->head, {{"head", desc.vocab, false}}, W));
        TLB_TRY(ld.vec("final.norm", &lm->final_norm, W));
        size_t part = 1;
        int kvh = 1;
        lm->ldp = lm->ldm = lm->ldu = 8;
        lm->lda = act_ld(W);
        for (const Layer &L : lm->layers) {
            lm->ldp = std::max(lm->ldp, act_ld(L.in.n));
            lm->ldm = std::max(lm->ldm, act_ld(L.out_width));
            lm->ldu = std::max(lm->ldu, act_ld(L.up.n));
            lm->lda = std::max(lm->lda, std::max(act_ld(L.out_width), act_ld(L.up.n)));
            if (L.d->mix.kind == MixerKind::Attention) {
                part = std::max(part, mix_attn_decode_partial_floats(attn_args(lm, L, nullptr, 0), B));
                kvh = std::max(kvh, L.d->mix.kv_heads);
            }
        }
        TLB_TRY(alloc(lm, &lm->proj, (size_t)B * lm->ldp));
        TLB_TRY(alloc(lm, &lm->mix, (size_t)B * lm->ldm));
        TLB_TRY(alloc(lm, &lm->up, (size_t)B * lm->ldu));
        TLB_TRY(alloc(lm, (char **)&lm->act, (size_t)B * lm->lda * 4));
        TLB_TRY(alloc(lm, &lm->partial, part));
        TLB_TRY(alloc(lm, &lm->counters, (size_t)B * kvh));
        return tlb_sync();
    };
    tlb_status st = build();
    if (st != TLB_OK) { layered_destroy(lm); return st; }
    *out = lm;
    return TLB_OK;
}

tlb_status layered_step(LayeredModel *lm, const int *token, const int *pos, const int *rope_pos, float *x, float *logits)
{
    const float eps = lm->desc.eps, off = lm->desc.norm_offset;
    bool first = true;
    for (const Layer &L : lm->layers) {
        DenseMatvecJob j;
        j.w = L.in; j.pro = DPRO_NORM; j.norm_w = L.norm1->f32(); j.norm_offset = off; j.eps = eps; j.out = lm->proj; j.x = x;
        if (first) { j.emb = lm->embed; j.token = token; j.x_out = x; }
        first = false;
        TLB_TRY(launch_dense_matvec(j));
        TLB_TRY(decode_mixer(lm, L, 1, pos, rope_pos, lm->mix, lm->ldm, true, true));
        j = DenseMatvecJob();
        j.w = L.o; j.x = lm->mix; j.out = x; j.resid_scale = L.ls1->f32();
        TLB_TRY(launch_dense_matvec(j));
        if (!L.up.w) continue;
        j = DenseMatvecJob();
        j.w = L.up; j.pro = DPRO_NORM; j.x = x; j.norm_w = L.norm2->f32(); j.norm_offset = off; j.eps = eps; j.out = lm->up;
        TLB_TRY(launch_dense_matvec(j));
        j = DenseMatvecJob();
        j.w = L.down; j.pro = DPRO_POLY; j.x = lm->up; j.poly = L.act->f32(); j.eps = eps; j.out = x; j.resid_scale = L.ls2->f32();
        TLB_TRY(launch_dense_matvec(j));
    }
    return layered_head(lm, x, 1, logits);
}

tlb_status layered_step_batch(LayeredModel *lm, const int *tokens, const int *pos, const int *rope_pos, int batch, float *x, float *logits)
{
    const int W = lm->desc.width;
    const float eps = lm->desc.eps, off = lm->desc.norm_offset;
    const bool f32 = lm->cfg.f32;
    TLB_TRY(launch_embed_bf16(tokens, lm->embed, W, lm->embed_ld, x, batch));
    for (const Layer &L : lm->layers) {
        const int ldw = act_ld(W), ldo = act_ld(L.out_width), ldf = act_ld(L.up.n);
        TLB_TRY(launch_norm_rows(x, batch, W, L.norm1->f32(), off, eps, lm->act, ldw, f32));
        TLB_TRY(rows_gemm(lm, L.in, lm->act, ldw, batch, lm->proj, lm->ldp, nullptr));
        TLB_TRY(decode_mixer(lm, L, batch, pos, rope_pos, lm->act, ldo, f32, false));
        TLB_TRY(rows_gemm(lm, L.o, lm->act, ldo, batch, x, W, L.ls1));
        if (!L.up.w) continue;
        TLB_TRY(launch_norm_rows(x, batch, W, L.norm2->f32(), off, eps, lm->act, ldw, f32));
        TLB_TRY(rows_gemm(lm, L.up, lm->act, ldw, batch, lm->up, lm->ldu, nullptr));
        TLB_TRY(launch_poly_rows(lm->up, batch, L.up.n, lm->ldu, L.act->f32(), eps, lm->act, ldf, f32));
        TLB_TRY(rows_gemm(lm, L.down, lm->act, ldf, batch, x, W, L.ls2));
    }
    return layered_head(lm, x, batch, logits);
}

tlb_status layered_prefill(LayeredModel *lm, int seq, const int32_t *tokens, int T, int pos0, int rope0, int rope_step, const int32_t *want,
                           int n_want, float *rows_out)
{
    const int W = lm->desc.width;
    const float eps = lm->desc.eps, off = lm->desc.norm_offset;
    const bool f32 = lm->cfg.f32;
    const size_t es = f32 ? 4 : 2;
    Rows ws;
    int *ids;
    float *x, *proj, *u, *o, *dly = nullptr;
    float2 *look = nullptr;
    void *act, *th = nullptr;
    size_t n_dly = 0, n_th = 0, n_look = 0;
    for (const Layer &L : lm->layers)
        if (L.d->mix.kind == MixerKind::GeneralDelta) { n_dly = std::max(n_dly, (size_t)L.w2.n); n_th = std::max(n_th, (size_t)L.w2.k); n_look = std::max(n_look, (size_t)L.d->mix.heads); }
    TLB_TRY(ws.get(&ids, ((size_t)T + std::max(n_want, 1)) * sizeof(int)));
    TLB_TRY(ws.get(&x, (size_t)T * W * 4));
    TLB_TRY(ws.get(&proj, (size_t)T * lm->ldp * 4));
    TLB_TRY(ws.get(&u, (size_t)T * lm->ldu * 4));
    TLB_TRY(ws.get(&o, (size_t)T * lm->ldm * 4));
    TLB_TRY(ws.get(&act, (size_t)T * lm->lda * es));
    if (n_dly) { TLB_TRY(ws.get(&dly, (size_t)T * n_dly * 4)); TLB_TRY(ws.get(&th, (size_t)T * n_th * es)); TLB_TRY(ws.get(&look, (size_t)scan_look_ld(T) * n_look * sizeof(float2))); }
    // pageable sources: staged before the calls return
    TLB_CUDA(cudaMemcpyAsync(ids, tokens, (size_t)T * sizeof(int), cudaMemcpyHostToDevice, ctx()->stream));
    if (n_want) TLB_CUDA(cudaMemcpyAsync(ids + T, want, (size_t)n_want * sizeof(int), cudaMemcpyHostToDevice, ctx()->stream));
    TLB_TRY(launch_embed_bf16(ids, lm->embed, W, lm->embed_ld, x, T));
    for (const Layer &L : lm->layers) {
        const int ldp = lm->ldp, ldw = act_ld(W), lda = act_ld(L.out_width), ldf = act_ld(L.up.n);
        TLB_TRY(launch_norm_rows(x, T, W, L.norm1->f32(), off, eps, act, ldw, f32));
        TLB_TRY(rows_gemm(lm, L.in, act, ldw, T, proj, ldp, nullptr));
        if (L.d->mix.kind == MixerKind::Attention) {
            TLB_TRY(launch_mix_attn_prefill(attn_args(lm, L, proj, ldp), seq, T, pos0, act, lda, f32));
        } else if (L.d->mix.kind == MixerKind::Retention) {
            TLB_TRY(launch_retention_prefill(recur_args(lm, L, proj, ldp), seq, T, pos0, rope0, rope_step, o, act, lda, f32));
        } else {
            TLB_TRY(launch_tanh_split(proj + 5 * (size_t)L.w2.n, T, L.d->mix.rank, ldp, th, L.w2.k / 2, f32));
            TLB_TRY(rows_gemm(lm, L.w2, th, L.w2.k, T, dly, L.w2.n, nullptr));
            TLB_TRY(launch_delta_prefill(recur_args(lm, L, proj, ldp), seq, T, pos0, dly, look, o, act, lda, f32));
        }
        TLB_TRY(rows_gemm(lm, L.o, act, lda, T, x, W, L.ls1));
        if (!L.up.w) continue;
        TLB_TRY(launch_norm_rows(x, T, W, L.norm2->f32(), off, eps, act, ldw, f32));
        TLB_TRY(rows_gemm(lm, L.up, act, ldw, T, u, lm->ldu, nullptr));
        TLB_TRY(launch_poly_rows(u, T, L.up.n, lm->ldu, L.act->f32(), eps, act, ldf, f32));
        TLB_TRY(rows_gemm(lm, L.down, act, ldf, T, x, W, L.ls2));
    }
    if (n_want) TLB_TRY(launch_gather_rows(x, W, ids + T, n_want, rows_out));
    return TLB_OK;
}

tlb_status layered_head(LayeredModel *lm, const float *rows, int n, float *logits)
{
    const int W = lm->desc.width, V = lm->desc.vocab;
    if (n == 1) {
        DenseMatvecJob j;
        j.w = lm->head; j.pro = DPRO_NORM; j.x = rows; j.norm_w = lm->final_norm->f32(); j.norm_offset = lm->desc.norm_offset; j.eps = lm->desc.eps; j.out = logits;
        return launch_dense_matvec(j);
    }
    const int ld = act_ld(W);
    Rows ws;
    void *act;
    TLB_TRY(ws.get(&act, (size_t)n * ld * (lm->cfg.f32 ? 4 : 2)));
    TLB_TRY(launch_norm_rows(rows, n, W, lm->final_norm->f32(), lm->desc.norm_offset, lm->desc.eps, act, ld, lm->cfg.f32));
    return rows_gemm(lm, lm->head, act, ld, n, logits, V, nullptr);
}

uint64_t layered_weight_bytes(const LayeredModel *lm) { return lm->weight_bytes - (uint64_t)lm->desc.vocab * lm->desc.width * 2 + (uint64_t)lm->desc.width * 2; }

uint64_t layered_state_bytes(const LayeredModel *lm, int ctx_len)
{
    uint64_t b = 0;
    for (const Layer &L : lm->layers) {
        const MixerDesc &x = L.d->mix;
        if (x.kind == MixerKind::Attention)
            b += (uint64_t)std::min(ctx_len, x.window > 0 ? x.window : ctx_len) * x.kv_heads * (x.dim + x.vdim) * (lm->cfg.f32 ? 4 : 2);
        else
            b += 2ull * x.heads * x.vdim * mix_recur_ld(x.dim) * 4;      // read and written
    }
    return b;
}

int layered_kernels_per_step(const LayeredModel *lm)
{
    int n = 1;
    for (const Layer &L : lm->layers) n += L.up.w ? 5 : 3;
    return n;
}

}  // namespace tlb
