// Registry of the designs that are described by a config.json: name -> reader of its keys.  Host code only.
#include "model_desc.h"

#include <cmath>

namespace tlb {
namespace {

// Typed access with a message that names the key.
struct Keys {
    std::string where;
    tlb_status st = TLB_OK;
    void bad(const char *key, const char *what) { if (st == TLB_OK) st = fail(TLB_ERR_ARG, "config.json: %s.%s %s", where.c_str(), key, what); }
    static bool given(const JVal &v, const char *key) { const JVal *o = v.get(key); return o && !o->is(JVal::NUL); }
    const JVal *obj(const JVal &v, const char *key)
    {
        const JVal *o = v.get(key);
        if (!o || !o->is(JVal::OBJ)) { bad(key, "is missing or not an object"); return nullptr; }
        return o;
    }
    double num(const JVal &v, const char *key)
    {
        const JVal *o = v.get(key);
        if (!o || !o->is(JVal::NUM) || !std::isfinite(o->num)) { bad(key, "is missing or not a number"); return 0.0; }
        return o->num;
    }
    int size(const JVal &v, const char *key, int64_t max = 1 << 24)
    {
        const double d = num(v, key);
        if (st != TLB_OK) return 0;
        if (d < 1 || d > (double)max || d != std::floor(d)) { bad(key, "is not a usable size"); return 0; }
        return (int)d;
    }
    std::string str(const JVal &v, const char *key)
    {
        const JVal *o = v.get(key);
        if (!o || !o->is(JVal::STR)) { bad(key, "is missing or not a string"); return ""; }
        return o->str;
    }
};

// the rotation of the leading dimensions of a vector of `size`
void read_rotation(Keys &k, const JVal &mixer, int size, MixerDesc *d)
{
    const JVal *rot = k.obj(mixer, "rot");
    if (!rot) return;
    d->rot_dims = k.size(*rot, "dims");
    d->rot_base = k.num(*rot, "base");
    if (k.st == TLB_OK && (d->rot_dims % 2 || d->rot_dims > size || d->rot_base <= 0.0)) k.bad("rot", "needs an even number of dims within the head and a positive base");
    if (!Keys::given(*rot, "scaling")) return;
    const JVal *sc = k.obj(*rot, "scaling");
    if (!sc) return;
    RotScaling &r = d->rot_scaling;
    r.factor = k.num(*sc, "factor"); r.original = k.num(*sc, "original"); r.fast = k.num(*sc, "fast"); r.slow = k.num(*sc, "slow");
    if (k.st == TLB_OK && (r.factor <= 0.0 || r.original <= 0.0 || r.fast <= 0.0 || r.slow <= 0.0 || d->rot_base == 1.0)) k.bad("rot.scaling", "needs positive numbers and a base other than 1");
}

// a mixture of experts or a dense feed-forward of gated activations
void read_gated_ffn(Keys &k, const JVal &mlp, FfnAct dense, FfnAct expert, FfnDesc *f)
{
    const std::string kind = k.str(mlp, "kind");
    if (k.st != TLB_OK) return;
    if (kind == "dense") {
        f->ff = k.size(mlp, "ff");
        f->act = dense;
        return;
    }
    if (kind != "moe") { k.st = fail(TLB_ERR_TYPE, "config.json: %s has feed-forward kind '%s', which is not known", k.where.c_str(), kind.c_str()); return; }
    f->act = expert;
    if (const JVal *e = k.obj(mlp, "expert")) f->ff = k.size(*e, "ff");
    const JVal *r = k.obj(mlp, "router");
    if (!r) return;
    f->experts = k.size(*r, "experts", 1024);
    f->top = k.size(*r, "top", 64);
    f->router_scale = (float)k.num(*r, "scale");
    if (Keys::given(*r, "groups")) {
        if (const JVal *g = k.obj(*r, "groups")) { f->groups = k.size(*g, "count"); f->keep = k.size(*g, "keep"); }
    }
    if (Keys::given(mlp, "shared")) {
        if (const JVal *s = k.obj(mlp, "shared")) f->shared_ff = k.size(*s, "ff");
    }
    if (k.st != TLB_OK) return;
    if (f->experts % f->groups || f->keep > f->groups) k.bad("mlp.router.groups", "do not divide the experts");
    else if (f->top > f->keep * (f->experts / f->groups)) k.bad("mlp.router.top", "is more than the experts of the kept groups");
}

tlb_status parse_mukutar(const JVal &c, ModelDesc *out)
{
    Keys k;
    k.where = "model";
    out->vocab = k.size(c, "vocab");
    out->width = k.size(c, "width");
    if (const JVal *n = k.obj(c, "norm")) out->eps = (float)k.num(*n, "eps");
    out->norm_offset = 1.f;
    const JVal *layers = c.get("layers");
    if (k.st == TLB_OK && (!layers || !layers->is(JVal::ARR) || layers->arr.empty())) k.bad("layers", "is missing or empty");
    if (k.st != TLB_OK) return k.st;
    for (size_t i = 0; i < layers->arr.size(); i++) {
        const JVal &l = layers->arr[i];
        k.where = "layers[" + std::to_string(i) + "]";
        if (!l.is(JVal::OBJ)) { k.bad("", "is not an object"); return k.st; }
        LayerDesc d;
        d.layer_scale = true;
        const std::string type = k.str(l, "type");
        const JVal *mx = k.obj(l, "mixer");
        if (k.st != TLB_OK) return k.st;
        MixerDesc &m = d.mix;
        m.heads = k.size(*mx, "heads");
        m.dim = k.size(*mx, "dim", 4096);
        if (type == "attention") {
            m.kind = MixerKind::Attention;
            m.kv_heads = k.size(*mx, "kv_heads");
            m.vdim = k.size(*mx, "vdim", 4096);
            m.scale = (float)k.num(*mx, "scale");
            m.qkv_bias = m.log_distance_bias = m.sink = true;
            if (const JVal *mask = k.obj(*mx, "mask")) m.window = k.size(*mask, "size", INT32_MAX);
            if (k.st == TLB_OK && m.heads % m.kv_heads) k.bad("mixer.heads", "is not a multiple of kv_heads");
        } else if (type == "retention") {
            m.kind = MixerKind::Retention;
            m.kv_heads = m.heads;
            m.vdim = k.size(*mx, "vdim", 4096);
            read_rotation(k, *mx, m.dim, &m);
            const JVal *dec = mx->get("decay");
            if (k.st == TLB_OK && (!dec || !dec->is(JVal::ARR) || dec->arr.size() != (size_t)m.heads)) k.bad("mixer.decay", "is not a list with one number per head");
            if (k.st != TLB_OK) return k.st;
            for (const JVal &v : dec->arr) {
                if (!v.is(JVal::NUM)) { k.bad("mixer.decay", "holds something that is not a number"); return k.st; }
                m.decay.push_back((float)v.num);
            }
        } else if (type == "general_delta") {
            m.kind = MixerKind::GeneralDelta;
            m.kv_heads = m.heads;
            m.vdim = m.dim;
        } else {
            return fail(TLB_ERR_TYPE, "config.json: %s has mixer type '%s', which %s does not have", k.where.c_str(), type.c_str(), out->arch.c_str());
        }
        const JVal *mlp = l.get("mlp");
        if (mlp && !mlp->is(JVal::NUL)) {
            if (!mlp->is(JVal::OBJ)) k.bad("mlp", "is neither null nor an object");
            else {
                const std::string kind = k.str(*mlp, "kind");
                if (k.st == TLB_OK && kind != "dense") return fail(TLB_ERR_TYPE, "config.json: %s has feed-forward kind '%s', which %s does not have", k.where.c_str(), kind.c_str(), out->arch.c_str());
                d.ffn.ff = k.size(*mlp, "ff");
                d.ffn.act = FfnAct::PolyNorm;
            }
        }
        if (k.st != TLB_OK) return k.st;
        out->layers.push_back(std::move(d));
    }
    return k.st;
}

bool same_sizes(const LayerDesc &a, const LayerDesc &b)
{
    const MixerDesc &x = a.mix, &y = b.mix;
    const FfnDesc &f = a.ffn, &g = b.ffn;
    return x.kind == y.kind && x.heads == y.heads && x.dim == y.dim && x.vdim == y.vdim && x.rot_dim == y.rot_dim && x.kv_rank == y.kv_rank && x.q_rank == y.q_rank &&
           x.out_gate == y.out_gate && x.width == y.width && x.window == y.window && x.scale == y.scale && x.rot_dims == y.rot_dims && x.rot_base == y.rot_base &&
           x.rot_scaling == y.rot_scaling && f.ff == g.ff && f.act == g.act && f.experts == g.experts && f.top == g.top && f.groups == g.groups && f.keep == g.keep &&
           f.router_scale == g.router_scale && f.shared_ff == g.shared_ff;
}

tlb_status parse_rukedra(const JVal &c, ModelDesc *out)
{
    Keys k;
    k.where = "model";
    out->vocab = k.size(c, "vocab");
    out->width = k.size(c, "width");
    if (const JVal *n = k.obj(c, "norm")) { out->eps = (float)k.num(*n, "eps"); out->norm_groups = k.size(*n, "groups", 256); }
    if (k.st == TLB_OK && out->width % out->norm_groups) k.bad("norm.groups", "does not divide the width");
    if (Keys::given(c, "logit_softcap")) {
        out->logit_softcap = (float)k.num(c, "logit_softcap");
        if (k.st == TLB_OK && out->logit_softcap <= 0.f) k.bad("logit_softcap", "is not positive");
    }
    const JVal *layers = c.get("layers");
    if (k.st == TLB_OK && (!layers || !layers->is(JVal::ARR) || layers->arr.empty())) k.bad("layers", "is missing or empty");
    if (k.st != TLB_OK) return k.st;
    for (size_t i = 0; i < layers->arr.size(); i++) {
        const JVal &l = layers->arr[i];
        k.where = "layers[" + std::to_string(i) + "]";
        if (!l.is(JVal::OBJ)) { k.bad("", "is not an object"); return k.st; }
        LayerDesc d;
        d.post_norm = d.resid_gate = true;
        const std::string type = k.str(l, "type");
        const JVal *mx = k.obj(l, "mixer");
        if (k.st != TLB_OK) return k.st;
        MixerDesc &m = d.mix;
        if (type == "latent_attention" || type == "latent_attention_2") {
            m.kind = MixerKind::Latent;
            m.heads = m.kv_heads = k.size(*mx, "heads");
            m.dim = k.size(*mx, "dim", 4096);
            m.rot_dim = k.size(*mx, "rot_dim", 4096);
            m.vdim = k.size(*mx, "vdim", 4096);
            m.kv_rank = k.size(*mx, "kv_rank", 65536);
            m.scale = (float)k.num(*mx, "scale");
            read_rotation(k, *mx, m.rot_dim, &m);
            if (type == "latent_attention") {
                m.q_rank = k.size(*mx, "q_rank", 65536);
                m.out_gate = true;
                if (const JVal *mask = k.obj(*mx, "mask")) m.window = k.size(*mask, "size", INT32_MAX);
            }
        } else if (type == "mingru") {
            m.kind = MixerKind::MinGru;
            m.width = k.size(*mx, "width");
        } else {
            return fail(TLB_ERR_TYPE, "config.json: %s has mixer type '%s', which %s does not have", k.where.c_str(), type.c_str(), out->arch.c_str());
        }
        const JVal *mlp = l.get("mlp");
        if (k.st == TLB_OK && mlp && !mlp->is(JVal::NUL)) {
            if (!mlp->is(JVal::OBJ)) k.bad("mlp", "is neither null nor an object");
            else read_gated_ffn(k, *mlp, FfnAct::GeluTanhGlu, FfnAct::SiluGlu, &d.ffn);
        }
        if (Keys::given(l, "weights_of")) {
            const double j = k.num(l, "weights_of");
            if (k.st == TLB_OK && (j < 0 || j >= (double)layers->arr.size() || j != std::floor(j) || j == (double)i)) k.bad("weights_of", "is not another layer's number");
            d.weights_of = (int)j;
        }
        if (k.st != TLB_OK) return k.st;
        out->layers.push_back(std::move(d));
    }
    // a layer may name one that itself uses another's tensors: the owner is what the loader needs
    for (size_t i = 0; i < out->layers.size(); i++) {
        LayerDesc &d = out->layers[i];
        k.where = "layers[" + std::to_string(i) + "]";
        for (size_t hops = 0; d.weights_of >= 0 && out->layers[d.weights_of].weights_of >= 0; hops++) {
            if (hops > out->layers.size()) { k.bad("weights_of", "never reaches a layer with tensors"); return k.st; }
            d.weights_of = out->layers[d.weights_of].weights_of;
        }
        if (d.weights_of >= 0 && !same_sizes(d, out->layers[d.weights_of])) { k.bad("weights_of", "names a layer that differs from this one"); return k.st; }
    }
    return k.st;
}

struct Design { const char *name; tlb_status (*parse)(const JVal &config, ModelDesc *out); };
const Design kDesigns[] = {
    {"Mukutar", parse_mukutar},
    {"Rukedra", parse_rukedra},
};

}  // namespace

bool map_has_model_config(const tlb_map *m) { return tlb_map_meta_string(m, "config.json") != nullptr; }

tlb_status model_desc_from_map(const tlb_map *m, ModelDesc *out)
{
    const char *text = tlb_map_meta_string(m, "config.json");
    if (!text) return fail(TLB_ERR_ARG, "the tensor map holds no config.json");
    JReader r{text, text + strlen(text)};
    JVal root;
    if (!r.value(root) || !root.is(JVal::OBJ)) return fail(TLB_ERR_ARG, "config.json is not a JSON object");
    const JVal *a = root.get("architecture");
    if (!a || !a->is(JVal::STR)) return fail(TLB_ERR_ARG, "config.json names no architecture");
    for (const Design &d : kDesigns)
        if (a->str == d.name) {
            *out = ModelDesc();
            out->arch = a->str;
            return d.parse(root, out);
        }
    return fail(TLB_ERR_TYPE, "architecture '%s' is not known (GGUF Llama models and: Mukutar, Rukedra)", a->str.c_str());
}

}  // namespace tlb
