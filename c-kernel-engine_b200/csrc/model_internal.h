/* What every model family shares behind the ckb200_model_* API (model.c): the configuration, the token and position staging of a
 * step, its captured graph, and the table of functions a family supplies.  A family's own model struct starts with these fields
 * (an unnamed `struct CKB200Model` member). */
#ifndef CKB200_MODEL_INTERNAL_H
#define CKB200_MODEL_INTERNAL_H

#include <cuda_runtime_api.h>
#include <stddef.h>
#include <stdint.h>

#include "../../include/ckb200_model.h"

typedef struct CkbModelFamily {
    const char *name;
    int (*claims)(const char *spec);                          /* does ckb200_model_open's spec name a model of this family? */
    CKB200Model *(*open)(const char *spec, int batch);
    void (*destroy)(CKB200Model *m);                          /* the family's own memory (the shared part is released by the caller) */
    int (*prepare)(CKB200Model *m, void *st);                 /* before a step is enqueued, outside any capture (may be NULL) */
    int (*issue_step)(CKB200Model *m, void *st);              /* one token per sequence: tokens_dev -> logits, position + 1 */
    /* `count` tokens per sequence in batched passes, logits of the wanted ones to the host; -1: not handled, the caller steps token by token */
    int (*extend)(CKB200Model *m, const int32_t *tokens, int count, const int32_t *want, int n_want, float *logits_host);
    int (*clear_state)(CKB200Model *m, void *st);             /* caches and recurrent state of all sequences, back to an empty context */
    int (*can_set_pos)(const CKB200Model *m);                 /* NULL: the position may be moved freely (nothing but indexed caches) */
    size_t (*step_weight_bytes)(const CKB200Model *m);        /* weight bytes one step streams */
} CkbModelFamily;

struct CKB200Model {
    CKB200ModelConfig c;
    const CkbModelFamily *family;
    int32_t *tokens_dev, *pos_dev;
    int32_t *tokens_pinned;
    int host_pos;           /* mirror of *pos_dev as of the last enqueued step (decode refuses to run past the context) */
    float *logits;          /* [batch][vocab] of the last step */
    cudaGraphExec_t graph;
    int graph_ready;
    cudaEvent_t ev_tokens;  /* the last copy out of tokens_pinned: the next call waits for it before it overwrites the buffer */
    int tokens_in_flight;
};

extern const CkbModelFamily ckb_family_kquant, ckb_family_stack;

/* token and position staging and the logits rows of `m` (its config is set); 0 on success */
int ckb_model_init_shared(struct CKB200Model *m);

#endif
