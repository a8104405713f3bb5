/* config.json of a layer-stack model -> StackConfig.  "architecture" picks a design from a table (which mixers it may use); every size and
 * constant comes from the file, and what is missing or makes no sense is refused with a message. */
#include <math.h>
#include <stdlib.h>
#include <string.h>

#include "json_mini.h"
#include "launch.h"
#include "layer_stack.h"
#include "mixers.h"

/* a design: its name in config.json, its layer types, the form of its layers, and where it differs in embedding and output */
typedef struct { const char *architecture; unsigned types; int form, tied, embed_scaled, capped; } StackDesign;
enum { TYPE_RETENTION = 0, TYPE_LATENT_ATTENTION, TYPE_CHANNEL_DELTA, TYPE_PARALLEL, TYPE_WKV, TYPES };
static const StackDesign g_designs[] = {
    { .architecture = "Puzevik", .types = 1u << TYPE_RETENTION | 1u << TYPE_LATENT_ATTENTION | 1u << TYPE_CHANNEL_DELTA, .form = STACK_PARALLEL, .embed_scaled = 1 },
    { .architecture = "Sipadra", .types = 1u << TYPE_PARALLEL | 1u << TYPE_WKV, .form = STACK_OUTPUT_NORM, .tied = 1, .capped = 1 },
};
/* a layer type: its mixers, and for two side by side where each is described and what its tensors are called */
static const struct { const char *name; int arms, mixer[STACK_ARMS]; const char *key[STACK_ARMS], *prefix[STACK_ARMS], *scale[STACK_ARMS]; } g_types[TYPES] = {
    [TYPE_RETENTION] = { "retention", 1, { STACK_RETENTION }, { NULL }, { "mix." }, { NULL } },
    [TYPE_LATENT_ATTENTION] = { "latent_attention", 1, { STACK_LATENT_ATTENTION }, { NULL }, { "mix." }, { NULL } },
    [TYPE_CHANNEL_DELTA] = { "channel_delta", 1, { STACK_CHANNEL_DELTA }, { NULL }, { "mix." }, { NULL } },
    [TYPE_PARALLEL] = { "parallel", 2, { STACK_WINDOW_ATTENTION, STACK_LIGHTNING }, { "left", "right" }, { "mix.left.", "mix.right." }, { "left_scale", "right_scale" } },
    [TYPE_WKV] = { "wkv", 1, { STACK_WKV }, { NULL }, { "mix." }, { NULL } },
};

static int positive(const JsonValue *obj, const char *key, int *out, const char *where)
{
    const JsonValue *v = json_get(obj, key);
    const double d = json_num(v, 0);
    if (!v || v->type != JSON_NUMBER || !(d >= 1 && d < 2147483647.0) || d != (double)(int)d) return ckb_fail(CKB_ERR_SHAPE, "config: %s needs a positive integer '%s'", where, key);
    *out = (int)d;
    return 0;
}

static int number(const JsonValue *obj, const char *key, double *out, const char *where)
{
    const JsonValue *v = json_get(obj, key);
    if (!v || v->type != JSON_NUMBER) return ckb_fail(CKB_ERR_SHAPE, "config: %s needs a number '%s'", where, key);
    *out = v->num;
    return 0;
}

static int rotation(StackMixer *x, const JsonValue *mixer, int max_dims, const char *where)
{
    const JsonValue *rot = json_get(mixer, "rot"), *yarn = json_get(rot, "scaling");
    if (positive(rot, "dims", &x->rot_dims, where) || number(rot, "base", &x->rot_base, where)) return CKB_ERR_SHAPE;
    if (x->rot_dims % 2 || x->rot_dims > max_dims || !(x->rot_base > 0)) return ckb_fail(CKB_ERR_SHAPE, "config: %s: rotation of %d dimensions out of %d", where, x->rot_dims, max_dims);
    if (!yarn || yarn->type != JSON_OBJECT) return 0;
    if (number(yarn, "factor", &x->yarn_factor, where) || number(yarn, "fast", &x->yarn_fast, where) || number(yarn, "slow", &x->yarn_slow, where) ||
        number(yarn, "original", &x->yarn_original, where))
        return CKB_ERR_SHAPE;
    if (!(x->yarn_factor > 0 && x->yarn_fast > 0 && x->yarn_slow > 0 && x->yarn_original > 0 && x->rot_base > 1))
        return ckb_fail(CKB_ERR_SHAPE, "config: %s: scaling of the rotation needs positive numbers and a base above 1", where);
    return 0;
}

/* YaRN: pairs that turn fast inside the original context keep their step, slow ones are stretched by the factor, with a ramp between the
 * pairs that make `fast` and `slow` turns */
float ckb_stack_frequencies(const StackMixer *x, float *freq)
{
    const int dims = x->rot_dims;
    double lo = 0, hi = 0;
    if (x->yarn_factor > 0) {
        const double per = dims / (2 * log(x->rot_base)), two_pi = 6.283185307179586476925;
        lo = floor(per * log(x->yarn_original / (two_pi * x->yarn_fast)));
        hi = ceil(per * log(x->yarn_original / (two_pi * x->yarn_slow)));
        if (lo < 0) lo = 0;
        if (hi > dims - 1) hi = dims - 1;
    }
    for (int i = 0; i < dims / 2; ++i) {
        const double f = pow(x->rot_base, -2.0 * i / dims);
        double ramp = 0;
        if (x->yarn_factor > 0) {
            ramp = (i - lo) / (hi - lo > 0.001 ? hi - lo : 0.001);
            ramp = ramp < 0 ? 0 : (ramp > 1 ? 1 : ramp);
        }
        freq[i] = (float)(ramp > 0 ? f / x->yarn_factor * ramp + f * (1 - ramp) : f);
    }
    return x->yarn_factor > 0 ? (float)(0.1 * log(x->yarn_factor) + 1) : 1.0f;
}

static int decays(StackMixer *x, const JsonValue *mx, const char *type)
{
    const JsonValue *decay = json_get(mx, "decay");
    if (json_len(decay) != x->heads) return ckb_fail(CKB_ERR_SHAPE, "config: %s needs one decay per head", type);
    x->decay_host = (float *)malloc((size_t)x->heads * sizeof(float));
    if (!x->decay_host) return ckb_fail(CKB_ERR_STATE, "config: out of memory");
    for (int h = 0; h < x->heads; ++h) x->decay_host[h] = (float)json_num(json_at(decay, h), 0);
    return 0;
}

static int grouped(StackMixer *x, const JsonValue *mx, const char *type)
{
    if (positive(mx, "kv_heads", &x->kv_heads, type)) return CKB_ERR_SHAPE;
    return x->heads % x->kv_heads ? ckb_fail(CKB_ERR_SHAPE, "config: %s: %d heads over %d key heads", type, x->heads, x->kv_heads) : 0;
}

static int read_mixer(StackMixer *x, const JsonValue *mx, const char *type)
{
    double scale = 0;
    if (positive(mx, "heads", &x->heads, type) || positive(mx, "dim", &x->dim, type)) return CKB_ERR_SHAPE;
    x->vdim = x->dim;
    if (x->type != STACK_WKV && positive(mx, "vdim", &x->vdim, type)) return CKB_ERR_SHAPE;
    x->kv_heads = x->heads;
    switch (x->type) {
        case STACK_RETENTION:
            if (rotation(x, mx, x->dim, type) || decays(x, mx, type)) return CKB_ERR_SHAPE;
            break;
        case STACK_LATENT_ATTENTION:
            if (positive(mx, "q_rank", &x->q_rank, type) || positive(mx, "kv_rank", &x->kv_rank, type) || positive(mx, "rot_dim", &x->rot_dim, type) ||
                number(mx, "scale", &scale, type) || rotation(x, mx, x->rot_dim, type))
                return CKB_ERR_SHAPE;
            if (x->rot_dims != x->rot_dim) return ckb_fail(CKB_ERR_SHAPE, "config: %s rotates %d of its %d rotated dimensions", type, x->rot_dims, x->rot_dim);
            break;
        case STACK_CHANNEL_DELTA:
            if (grouped(x, mx, type) || positive(mx, "conv", &x->taps, type)) return CKB_ERR_SHAPE;
            break;
        case STACK_WINDOW_ATTENTION:
            if (grouped(x, mx, type) || number(mx, "scale", &scale, type) || rotation(x, mx, x->dim, type) || positive(json_get(mx, "mask"), "size", &x->window, type)) return CKB_ERR_SHAPE;
            if (x->dim > 256 || x->vdim > 256) return ckb_fail(CKB_ERR_LIMIT, "config: %s: head size %d, values of %d", type, x->dim, x->vdim);
            break;
        case STACK_LIGHTNING:
            if (decays(x, mx, type)) return CKB_ERR_SHAPE;
            break;
    }
    x->scale = (float)scale;
    x->a_rank = (int)json_num(json_get(mx, "a_rank"), 0);
    x->g_rank = (int)json_num(json_get(mx, "g_rank"), 0);
    if (x->type != STACK_LATENT_ATTENTION && x->type != STACK_WINDOW_ATTENTION && !ckb_recur_dp(x->dim)) return ckb_fail(CKB_ERR_LIMIT, "config: %s: head size %d", type, x->dim);
    return 0;
}

static int read_layer(StackLayer *l, const JsonValue *e, unsigned allowed)
{
    const char *name = json_str(json_get(e, "type"), "");
    const JsonValue *mx = json_get(e, "mixer"), *mlp = json_get(e, "mlp");
    int type = -1;
    for (int i = 0; i < TYPES; ++i)
        if (!strcmp(name, g_types[i].name) && (allowed >> i & 1)) type = i;
    if (type < 0) return ckb_fail(CKB_ERR_SHAPE, "config: unknown layer type '%s'", name);
    l->arms = g_types[type].arms;
    for (int i = 0; i < l->arms; ++i) {
        StackMixer *x = &l->mix[i];
        const char *key = g_types[type].key[i];
        double scale = 1;
        x->type = g_types[type].mixer[i];
        x->prefix = g_types[type].prefix[i];
        if (g_types[type].scale[i] && number(mx, g_types[type].scale[i], &scale, name)) return CKB_ERR_SHAPE;
        x->out_scale = (float)scale;
        const int rc = read_mixer(x, key ? json_get(mx, key) : mx, key ? key : name);
        if (rc) return rc;
    }
    if (mlp && mlp->type == JSON_OBJECT) {
        const char *kind = json_str(json_get(mlp, "kind"), "");
        if (strcmp(kind, "dense")) return ckb_fail(CKB_ERR_SHAPE, "config: unknown feed-forward '%s'", kind);
        if (positive(mlp, "ff", &l->ff, "mlp")) return CKB_ERR_SHAPE;
    }
    return 0;
}

void ckb_stack_config_free(StackConfig *c)
{
    for (int i = 0; c->layers && i < c->n_layers; ++i)
        for (int k = 0; k < STACK_ARMS; ++k) free(c->layers[i].mix[k].decay_host);
    free(c->layers);
    memset(c, 0, sizeof *c);
}

int ckb_stack_config_read(const char *path, StackConfig *out)
{
    char err[160] = "";
    memset(out, 0, sizeof *out);
    JsonValue *root = json_parse_file(path, err, sizeof err);
    if (!root) return ckb_fail(CKB_ERR_STATE, "config: %s: %s", path, err);
    const char *arch = json_str(json_get(root, "architecture"), "");
    const StackDesign *design = NULL;
    for (size_t i = 0; i < sizeof g_designs / sizeof g_designs[0]; ++i)
        if (!strcmp(arch, g_designs[i].architecture)) design = &g_designs[i];
    const JsonValue *layers = json_get(root, "layers");
    double eps = 0, scale = 1, cap = 0;
    int rc = design ? 0 : ckb_fail(CKB_ERR_STATE, "config: no design '%s'", arch);
    if (!rc) rc = positive(root, "width", &out->width, "the model");
    if (!rc) rc = positive(root, "vocab", &out->vocab, "the model");
    if (!rc) rc = number(json_get(root, "norm"), "eps", &eps, "norm");
    if (!rc && design->embed_scaled) rc = number(json_get(root, "embedding"), "scale", &scale, "embedding");
    if (!rc && design->capped) rc = number(root, "logit_softcap", &cap, "the model");
    if (!rc && design->capped && !(cap > 0)) rc = ckb_fail(CKB_ERR_SHAPE, "config: logit_softcap must be positive");
    if (!rc && (!layers || layers->type != JSON_ARRAY || !layers->count)) rc = ckb_fail(CKB_ERR_SHAPE, "config: no layers");
    if (!rc) {
        out->eps = (float)eps;
        out->embed_scale = (float)scale;
        out->logit_cap = (float)cap;
        out->form = design->form;
        out->tied = design->tied;
        out->n_layers = layers->count;
        out->layers = (StackLayer *)calloc((size_t)layers->count, sizeof(StackLayer));
        if (!out->layers) rc = ckb_fail(CKB_ERR_STATE, "config: out of memory");
        for (int i = 0; !rc && i < layers->count; ++i) rc = read_layer(&out->layers[i], json_at(layers, i), design->types);
    }
    json_free(root);
    if (rc) ckb_stack_config_free(out);
    return rc;
}
