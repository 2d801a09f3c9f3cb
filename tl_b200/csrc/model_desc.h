// What a model folder (config.json + model.safetensors) describes: a decoder as a list of layers, each with one of several
// mixers and an optional feed-forward.  model_registry.cu turns the config of a known design into a ModelDesc; layered.cu
// runs any ModelDesc.  Everything that may differ between designs is a field here, not a branch on a design's name.
#pragma once
#include <string>
#include <vector>

#include "json.h"
#include "tlb_internal.h"

namespace tlb {

enum class MixerKind {
    Attention,      // softmax attention over a KV cache
    Retention,      // linear attention with a fixed decay per head
    GeneralDelta,   // generalised delta rule: decay per key channel, removal along the unit key
    Latent,         // softmax attention over a cache of latents and one shared rotated key part per token
    MinGru,         // gated recurrence per channel whose gates read only the current token
};

// Slower angles for pairs that turn seldom within `original` positions (YaRN); factor 0: none.
struct RotScaling {
    double factor = 0.0, original = 0.0, fast = 0.0, slow = 0.0;
    bool operator==(const RotScaling &o) const { return factor == o.factor && original == o.original && fast == o.fast && slow == o.slow; }
};

struct MixerDesc {
    MixerKind kind = MixerKind::Attention;
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    // Attention
    float scale = 1.f;          // factor on q . k
    int window = 0;             // keys a query sees, itself included; 0: all before it
    bool qkv_bias = false;      // q, k, v projections have biases
    bool log_distance_bias = false;   // score -= r1[h] * ln(1 + r2[h] * distance)
    bool sink = false;          // exp(sink[h]) joins the softmax denominator
    // Retention (rotate-half pairs), Latent (pairs of neighbours)
    int rot_dims = 0;           // leading dimensions of q and k (Latent: of the rotated part) that turn; 0: none
    double rot_base = 0.0;
    RotScaling rot_scaling;
    std::vector<float> decay;   // Retention: per head
    // GeneralDelta
    int rank = 0;               // inner size of the decay's two-step projection (from the tensor's shape)
    // Latent: `dim` unrotated and `rot_dim` shared rotated key dimensions; also scale and window above
    int rot_dim = 0, kv_rank = 0;
    int q_rank = 0;             // size of the latent the queries go through; 0: projected directly
    bool out_gate = false;      // every output element times a sigmoid of a projection
    // MinGru
    int width = 0;
};

enum class FfnAct { PolyNorm, SiluGlu, GeluTanhGlu };

struct FfnDesc {
    int ff = 0;                 // 0: the layer has no feed-forward; mixture of experts: of one expert
    FfnAct act = FfnAct::PolyNorm;
    // mixture of experts
    int experts = 0;            // 0: dense
    int top = 0, groups = 1, keep = 1;
    float router_scale = 1.f;
    int shared_ff = 0;          // 0: no shared expert
};

struct LayerDesc {
    MixerDesc mix;
    FfnDesc ffn;
    bool layer_scale = false;   // per-channel factors on what the mixer and the feed-forward add to the residual
    bool post_norm = false;     // a second norm on what the mixer and the feed-forward add
    bool resid_gate = false;    // ... which is first multiplied by a sigmoid of a projection of the sublayer's input
    int weights_of = -1;        // the layer whose tensors this one uses (with a cache or state of its own)
};

struct ModelDesc {
    std::string arch;
    int vocab = 0, width = 0;
    float eps = 0.f;
    float norm_offset = 0.f;    // added to the stored weight of the width norms (1: stored around zero)
    int norm_groups = 1;        // equal parts of the width, each over its own root mean square
    float logit_softcap = 0.f;  // > 0: logits go through cap * tanh(. / cap)
    std::vector<LayerDesc> layers;
};

// The design named by the map's config.json, parsed and checked.  TLB_ERR_ARG when the map has none or it is malformed,
// TLB_ERR_TYPE for a design that is not registered.
tlb_status model_desc_from_map(const tlb_map *m, ModelDesc *out);
bool map_has_model_config(const tlb_map *m);
// tensors as the folder holds them (gguf.cu): the bf16 matrix itself, not widened; null when absent or of another type
const tlb_tensor *map_raw_bf16(const tlb_map *m, const std::string &name);
bool map_has(const tlb_map *m, const std::string &name);

// ---- the model as a session runs it (layered.cu) -----------------------------------------------------------------
struct LayeredModel;
struct LayeredCfg {
    int max_seq = 0, batch = 1;
    bool f32 = false;           // all products in 32 bits and f32 caches; otherwise bf16 operands, f16 caches
};
tlb_status layered_create(LayeredModel **out, const ModelDesc &desc, tlb_map *m, const LayeredCfg &cfg);
void layered_destroy(LayeredModel *lm);
// One token of sequence 0: *token at row *pos (rotated by *rope_pos), read on the device; the residual goes to x [width], the
// logits to logits [vocab].
tlb_status layered_step(LayeredModel *lm, const int *token, const int *pos, const int *rope_pos, float *x, float *logits);
// One token of every sequence (arrays on the device), residual rows in x [batch, width], logits [batch, vocab].
tlb_status layered_step_batch(LayeredModel *lm, const int *tokens, const int *pos, const int *rope_pos, int batch, float *x, float *logits);
// T tokens (host) of one sequence behind its first pos0; the residual rows of tokens want[i] (offsets from the first) go to
// rows_out [n_want, width].
tlb_status layered_prefill(LayeredModel *lm, int seq, const int32_t *tokens, int T, int pos0, int rope0, int rope_step, const int32_t *want,
                           int n_want, float *rows_out);
// final norm + head of n residual rows
tlb_status layered_head(LayeredModel *lm, const float *rows, int n, float *logits);
uint64_t layered_weight_bytes(const LayeredModel *lm);
uint64_t layered_state_bytes(const LayeredModel *lm, int ctx_len);   // cache rows and recurrent state one step touches
int layered_kernels_per_step(const LayeredModel *lm);

}  // namespace tlb
