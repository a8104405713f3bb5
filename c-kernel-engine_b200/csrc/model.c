/* The ckb200_model_* API shared by every model family: which family opens a spec, token staging, the captured decode step and its
 * replay, prompt passes, position and reset (the counterpart of the reference's ck_model_* calls around the generated ck_decode /
 * ck_prefill, version/v7/scripts/codegen_v7.py:1282-1426).  What a step consists of is the family's business (model_internal.h). */
#include <cuda_runtime_api.h>
#include <stdint.h>
#include <stdlib.h>
#include <string.h>

#include "../../include/ckb200.h"
#include "launch.h"
#include "model_internal.h"
#include "runtime.h"

/* asked in this order; a library built with fewer families has NULL entries */
extern const CkbModelFamily ckb_family_kquant __attribute__((weak));
extern const CkbModelFamily ckb_family_stack __attribute__((weak));
static const CkbModelFamily *const g_families[] = { &ckb_family_stack, &ckb_family_kquant };

CKB200Model *ckb200_model_open(const char *spec, int batch)
{
    if (!spec) { ckb_fail(CKB_ERR_STATE, "model_open: NULL spec"); return NULL; }
    for (size_t i = 0; i < sizeof g_families / sizeof g_families[0]; ++i)
        if (g_families[i] && g_families[i]->claims(spec)) return g_families[i]->open(spec, batch);
    ckb_fail(CKB_ERR_STATE, "model_open: no model family of this library takes '%s'", spec);
    return NULL;
}

int ckb_model_init_shared(struct CKB200Model *m)
{
    const size_t B = (size_t)m->c.batch;
    cudaStream_t st = ckb_stream(NULL);
    if (ckb_check_cuda((int)cudaMalloc((void **)&m->tokens_dev, B * sizeof(int32_t)), "cudaMalloc(tokens)") ||
        ckb_check_cuda((int)cudaMalloc((void **)&m->pos_dev, 256), "cudaMalloc(position)") ||
        ckb_check_cuda((int)cudaMalloc((void **)&m->logits, B * (size_t)m->c.vocab_size * sizeof(float)), "cudaMalloc(logits)") ||
        ckb_check_cuda((int)cudaHostAlloc((void **)&m->tokens_pinned, B * sizeof(int32_t), cudaHostAllocDefault), "cudaHostAlloc") ||
        ckb_check_cuda((int)cudaEventCreateWithFlags(&m->ev_tokens, cudaEventDisableTiming), "tokens event") ||
        ckb_check_cuda((int)cudaMemsetAsync(m->pos_dev, 0, 256, st), "zero position"))
        return CKB_ERR_CUDA;
    return 0;
}

void ckb200_model_free(CKB200Model *m)
{
    if (!m) return;
    cudaStreamSynchronize(ckb_stream(NULL));
    if (m->graph_ready) cudaGraphExecDestroy(m->graph);
    m->family->destroy(m);
    void *ptrs[] = { m->tokens_dev, m->pos_dev, m->logits };
    for (size_t i = 0; i < sizeof ptrs / sizeof ptrs[0]; ++i) if (ptrs[i]) cudaFree(ptrs[i]);
    if (m->tokens_pinned) cudaFreeHost(m->tokens_pinned);
    if (m->ev_tokens) cudaEventDestroy(m->ev_tokens);
    free(m);
}

const CKB200ModelConfig *ckb200_model_config(CKB200Model *m) { return m ? &m->c : NULL; }
const char *ckb200_model_family(CKB200Model *m) { return m ? m->family->name : NULL; }
float *ckb200_model_logits_device(CKB200Model *m) { return m ? m->logits : NULL; }
size_t ckb200_model_weight_bytes(CKB200Model *m) { return m ? m->family->step_weight_bytes(m) : 0; }

static int write_pos(CKB200Model *m, int pos)
{
    int32_t p = pos;
    cudaStream_t st = ckb_stream(NULL);
    if (ckb_check_cuda((int)cudaMemcpyAsync(m->pos_dev, &p, sizeof p, cudaMemcpyHostToDevice, st), "set pos")) return CKB_ERR_CUDA;
    if (ckb_check_cuda((int)cudaStreamSynchronize(st), "set pos")) return CKB_ERR_CUDA;
    m->host_pos = pos;
    return 0;
}

int ckb200_model_set_pos(CKB200Model *m, int pos)
{
    if (!m || pos < 0 || pos >= m->c.max_seq_len) return ckb_fail(CKB_ERR_STATE, "model_set_pos: %d outside [0, %d)", pos, m ? m->c.max_seq_len : 0);
    if (m->family->can_set_pos && !m->family->can_set_pos(m)) {
        /* a recurrent state has no positions to return to: only the empty context and the present position exist */
        if (pos == 0) return ckb200_model_reset(m);
        if (pos != m->host_pos) return ckb_fail(CKB_ERR_STATE, "model_set_pos: this model carries a recurrent state; it cannot move from %d to %d", m->host_pos, pos);
    }
    return write_pos(m, pos);
}

int ckb200_model_get_pos(CKB200Model *m)
{
    int32_t p = -1;
    if (!m) return -1;
    cudaStreamSynchronize(ckb_stream(NULL));
    cudaMemcpy(&p, m->pos_dev, sizeof p, cudaMemcpyDeviceToHost);
    return p;
}

int ckb200_model_reset(CKB200Model *m)
{
    if (!m) return CKB_ERR_STATE;
    const int rc = m->family->clear_state(m, ckb_stream(NULL));
    return rc ? rc : write_pos(m, 0);
}

/* ------------------------------------------------------------------ the decode step */

int ckb200_model_decode(CKB200Model *m, const int32_t *tokens, float *logits_host)
{
    if (!m || !tokens) return ckb_fail(CKB_ERR_STATE, "model_decode: NULL model or tokens");
    if (m->host_pos >= m->c.max_seq_len)
        return ckb_fail(CKB_ERR_LIMIT, "model_decode: position %d is past the context of %d tokens (reset or set_pos first)", m->host_pos, m->c.max_seq_len);
    cudaStream_t st = ckb_stream(NULL);
    const int B = m->c.batch;
    /* a call without logits_host returns while its step is still queued: the pinned staging buffer may only be reused once the
     * copy out of it has run */
    if (m->tokens_in_flight && ckb_check_cuda((int)cudaEventSynchronize(m->ev_tokens), "tokens staging")) return CKB_ERR_CUDA;
    memcpy(m->tokens_pinned, tokens, (size_t)B * sizeof(int32_t));
    if (ckb_check_cuda((int)cudaMemcpyAsync(m->tokens_dev, m->tokens_pinned, (size_t)B * sizeof(int32_t), cudaMemcpyHostToDevice, st), "tokens H2D")) return CKB_ERR_CUDA;
    if (ckb_check_cuda((int)cudaEventRecord(m->ev_tokens, st), "tokens event")) return CKB_ERR_CUDA;
    m->tokens_in_flight = 1;
    if (m->family->prepare) { const int rc = m->family->prepare(m, st); if (rc) return rc; }
    const int use_graph = ckb_tune_get("model_graph", 1);
    if (use_graph && !m->graph_ready) {
        /* this step runs eagerly: it sets per-kernel attributes (not allowed while capturing), and a step that advances a recurrent
         * state cannot be run twice.  Then the step is captured for the calls that follow. */
        int rc = m->family->issue_step(m, st);
        if (rc) return rc;
        if (ckb_check_cuda((int)cudaStreamSynchronize(st), "first step")) return CKB_ERR_CUDA;
        cudaGraph_t g = NULL;
        if (ckb_check_cuda((int)cudaStreamBeginCapture(st, cudaStreamCaptureModeThreadLocal), "begin capture")) return CKB_ERR_CUDA;
        rc = m->family->issue_step(m, st);
        const cudaError_t e = cudaStreamEndCapture(st, &g);
        if (rc || e != cudaSuccess || !g) {
            if (g) cudaGraphDestroy(g);
            return rc ? rc : ckb_check_cuda((int)e, "end capture");
        }
        const cudaError_t ei = cudaGraphInstantiate(&m->graph, g, 0);
        cudaGraphDestroy(g);
        if (ckb_check_cuda((int)ei, "graph instantiate")) return CKB_ERR_CUDA;
        m->graph_ready = 1;
    } else if (use_graph) {
        if (ckb_check_cuda((int)cudaGraphLaunch(m->graph, st), "graph launch")) return CKB_ERR_CUDA;
    } else {
        const int rc = m->family->issue_step(m, st);
        if (rc) return rc;
    }
    m->host_pos += 1;
    if (logits_host) {
        if (ckb_check_cuda((int)cudaMemcpyAsync(logits_host, m->logits, (size_t)B * m->c.vocab_size * sizeof(float), cudaMemcpyDeviceToHost, st), "logits D2H")) return CKB_ERR_CUDA;
        return ckb_sync_check(st, "model_decode");        /* a timed-out exchange must not come back as rc 0 with stale logits */
    }
    return 0;
}

/* ------------------------------------------------------------------ prompts and portions of prompts */

int ckb200_model_extend(CKB200Model *m, const int32_t *tokens, int count, const int32_t *want, int n_want, float *logits_host)
{
    if (!m || !tokens || count <= 0 || n_want < 0 || (n_want && (!want || !logits_host))) return ckb_fail(CKB_ERR_STATE, "model_extend: NULL or empty argument");
    if (m->host_pos + count > m->c.max_seq_len)
        return ckb_fail(CKB_ERR_LIMIT, "model_extend: %d tokens from position %d run past the context of %d tokens", count, m->host_pos, m->c.max_seq_len);
    for (int i = 0; i < n_want; ++i)
        if (want[i] < 0 || want[i] >= count || (i && want[i] <= want[i - 1])) return ckb_fail(CKB_ERR_STATE, "model_extend: wanted places must ascend inside the portion");
    if (m->family->prepare) { const int rc = m->family->prepare(m, ckb_stream(NULL)); if (rc) return rc; }
    if (count > 1) {
        const int rc = m->family->extend(m, tokens, count, want, n_want, logits_host);
        if (rc != -1) return rc;
    }
    const size_t B = (size_t)m->c.batch;
    int w = 0;
    for (int i = 0; i < count; ++i) {
        const int take = w < n_want && want[w] == i;
        const int rc = ckb200_model_decode(m, tokens + (size_t)i * B, take ? logits_host + (size_t)w * B * m->c.vocab_size : NULL);
        if (rc) return rc;
        w += take;
    }
    return 0;
}

int ckb200_model_prefill(CKB200Model *m, const int32_t *tokens, int count, float *logits_host)
{
    const int32_t last = count - 1;
    return ckb200_model_extend(m, tokens, count, &last, logits_host ? 1 : 0, logits_host);
}

/* Enqueue `steps` decode steps that keep feeding the same token ids (benchmark loop; no host sync). */
int ckb200_model_decode_repeat(CKB200Model *m, int steps)
{
    if (!m || !m->graph_ready) return ckb_fail(CKB_ERR_STATE, "model_decode_repeat: run model_decode once first");
    if (steps > m->c.max_seq_len - m->host_pos)
        return ckb_fail(CKB_ERR_LIMIT, "model_decode_repeat: %d steps from position %d run past the context of %d tokens", steps, m->host_pos, m->c.max_seq_len);
    cudaStream_t st = ckb_stream(NULL);
    for (int i = 0; i < steps; ++i)
        if (ckb_check_cuda((int)cudaGraphLaunch(m->graph, st), "graph launch")) return CKB_ERR_CUDA;
    m->host_pos += steps;
    return 0;
}
