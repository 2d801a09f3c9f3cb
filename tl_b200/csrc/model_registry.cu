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

void read_rotation(Keys &k, const JVal &mixer, MixerDesc *d)
{
    const JVal *rot = k.obj(mixer, "rot");
    if (!rot) return;
    d->rot_dims = k.size(*rot, "dims");
    d->rot_base = k.num(*rot, "base");
    if (k.st == TLB_OK && (d->rot_dims % 2 || d->rot_dims > d->dim || d->rot_base <= 0.0)) k.bad("rot", "needs an even number of dims within the head and a positive base");
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
            read_rotation(k, *mx, &m);
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

struct Design { const char *name; tlb_status (*parse)(const JVal &config, ModelDesc *out); };
const Design kDesigns[] = {
    {"Mukutar", parse_mukutar},
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
    return fail(TLB_ERR_TYPE, "architecture '%s' is not known (GGUF Llama models and: Mukutar)", a->str.c_str());
}

}  // namespace tlb
