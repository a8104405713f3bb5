/* config.json of a layer-stack model -> StackConfig.  "architecture" picks a design from a table (which mixers it may use); every size and
 * constant comes from the file, and what is missing or makes no sense is refused with a message. */
#include <stdlib.h>
#include <string.h>

#include "json_mini.h"
#include "launch.h"
#include "layer_stack.h"
#include "mixers.h"

/* a design: its name in config.json and its mixers.  Its layers are of the parallel form: one RMS norm whose output both the mixer and
 * the feed-forward read, both results added to the residual. */
typedef struct { const char *architecture; unsigned mixers; } StackDesign;
static const StackDesign g_designs[] = {
    { "Puzevik", 1u << STACK_RETENTION | 1u << STACK_LATENT_ATTENTION | 1u << STACK_CHANNEL_DELTA },
};
static const char *const g_mixer_names[STACK_MIXERS] = { "retention", "latent_attention", "channel_delta" };

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

static int rotation(StackLayer *l, const JsonValue *mixer, int max_dims, const char *where)
{
    const JsonValue *rot = json_get(mixer, "rot");
    if (positive(rot, "dims", &l->rot_dims, where) || number(rot, "base", &l->rot_base, where)) return CKB_ERR_SHAPE;
    if (l->rot_dims % 2 || l->rot_dims > max_dims || !(l->rot_base > 0)) return ckb_fail(CKB_ERR_SHAPE, "config: %s: rotation of %d dimensions out of %d", where, l->rot_dims, max_dims);
    return 0;
}

static int read_layer(StackLayer *l, const JsonValue *e, unsigned allowed)
{
    const char *type = json_str(json_get(e, "type"), "");
    const JsonValue *mx = json_get(e, "mixer"), *mlp = json_get(e, "mlp");
    l->type = -1;
    for (int i = 0; i < STACK_MIXERS; ++i)
        if (!strcmp(type, g_mixer_names[i]) && (allowed >> i & 1)) l->type = i;
    if (l->type < 0) return ckb_fail(CKB_ERR_SHAPE, "config: unknown layer type '%s'", type);
    if (positive(mx, "heads", &l->heads, type) || positive(mx, "dim", &l->dim, type) || positive(mx, "vdim", &l->vdim, type)) return CKB_ERR_SHAPE;
    l->kv_heads = l->heads;
    if (l->type == STACK_RETENTION) {
        const JsonValue *decay = json_get(mx, "decay");
        if (rotation(l, mx, l->dim, type)) return CKB_ERR_SHAPE;
        if (json_len(decay) != l->heads) return ckb_fail(CKB_ERR_SHAPE, "config: %s needs one decay per head", type);
        l->decay_host = (float *)malloc((size_t)l->heads * sizeof(float));
        if (!l->decay_host) return ckb_fail(CKB_ERR_STATE, "config: out of memory");
        for (int h = 0; h < l->heads; ++h) l->decay_host[h] = (float)json_num(json_at(decay, h), 0);
    } else if (l->type == STACK_LATENT_ATTENTION) {
        double scale = 0;
        if (positive(mx, "q_rank", &l->q_rank, type) || positive(mx, "kv_rank", &l->kv_rank, type) || positive(mx, "rot_dim", &l->rot_dim, type) ||
            number(mx, "scale", &scale, type) || rotation(l, mx, l->rot_dim, type))
            return CKB_ERR_SHAPE;
        if (l->rot_dims != l->rot_dim) return ckb_fail(CKB_ERR_SHAPE, "config: %s rotates %d of its %d rotated dimensions", type, l->rot_dims, l->rot_dim);
        l->scale = (float)scale;
    } else {
        if (positive(mx, "kv_heads", &l->kv_heads, type) || positive(mx, "conv", &l->taps, type)) return CKB_ERR_SHAPE;
        if (l->heads % l->kv_heads) return ckb_fail(CKB_ERR_SHAPE, "config: %s: %d heads over %d key heads", type, l->heads, l->kv_heads);
        l->a_rank = (int)json_num(json_get(mx, "a_rank"), 0);
        l->g_rank = (int)json_num(json_get(mx, "g_rank"), 0);
    }
    if (l->type != STACK_LATENT_ATTENTION && !ckb_recur_dp(l->dim)) return ckb_fail(CKB_ERR_LIMIT, "config: %s: head size %d", type, l->dim);
    if (mlp && mlp->type == JSON_OBJECT) {
        const char *kind = json_str(json_get(mlp, "kind"), "");
        if (strcmp(kind, "dense")) return ckb_fail(CKB_ERR_SHAPE, "config: unknown feed-forward '%s'", kind);
        if (positive(mlp, "ff", &l->ff, "mlp")) return CKB_ERR_SHAPE;
    }
    return 0;
}

void ckb_stack_config_free(StackConfig *c)
{
    for (int i = 0; c->layers && i < c->n_layers; ++i) free(c->layers[i].decay_host);
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
    double eps = 0, scale = 0;
    int rc = design ? 0 : ckb_fail(CKB_ERR_STATE, "config: no design '%s'", arch);
    if (!rc) rc = positive(root, "width", &out->width, "the model");
    if (!rc) rc = positive(root, "vocab", &out->vocab, "the model");
    if (!rc) rc = number(json_get(root, "norm"), "eps", &eps, "norm");
    if (!rc) rc = number(json_get(root, "embedding"), "scale", &scale, "embedding");
    if (!rc && (!layers || layers->type != JSON_ARRAY || !layers->count)) rc = ckb_fail(CKB_ERR_SHAPE, "config: no layers");
    if (!rc) {
        out->eps = (float)eps;
        out->embed_scale = (float)scale;
        out->n_layers = layers->count;
        out->layers = (StackLayer *)calloc((size_t)layers->count, sizeof(StackLayer));
        if (!out->layers) rc = ckb_fail(CKB_ERR_STATE, "config: out of memory");
        for (int i = 0; !rc && i < layers->count; ++i) rc = read_layer(&out->layers[i], json_at(layers, i), design->mixers);
    }
    json_free(root);
    if (rc) ckb_stack_config_free(out);
    return rc;
}
