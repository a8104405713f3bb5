/* safetensors reader over a memory-mapped file; every offset is checked against the file before it is handed out. */
#define _GNU_SOURCE
#include <fcntl.h>
#include <stdlib.h>
#include <string.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include "json_mini.h"
#include "launch.h"
#include "safetensors.h"

struct CkbSafetensors {
    uint8_t *map;
    size_t size, data0;
    JsonValue *head;
};

CkbSafetensors *ckb_st_open(const char *path)
{
    const int fd = open(path, O_RDONLY);
    if (fd < 0) { ckb_fail(CKB_ERR_STATE, "safetensors: cannot open %s", path); return NULL; }
    struct stat sb;
    CkbSafetensors *f = (CkbSafetensors *)calloc(1, sizeof *f);
    char err[160] = "file too short";
    if (f && fstat(fd, &sb) == 0 && sb.st_size >= 8) {
        f->size = (size_t)sb.st_size;
        void *p = mmap(NULL, f->size, PROT_READ, MAP_PRIVATE, fd, 0);
        f->map = p == MAP_FAILED ? NULL : (uint8_t *)p;
    }
    close(fd);
    if (f && f->map) {
        uint64_t n = 0;
        for (int i = 7; i >= 0; --i) n = n << 8 | f->map[i];
        if (n <= f->size - 8) {
            f->data0 = 8 + (size_t)n;
            f->head = json_parse((const char *)f->map + 8, (size_t)n, err, sizeof err);
        }
    }
    if (!f || !f->head || f->head->type != JSON_OBJECT) {
        ckb_fail(CKB_ERR_STATE, "safetensors: %s: %s", path, err);
        ckb_st_close(f);
        return NULL;
    }
    return f;
}

void ckb_st_close(CkbSafetensors *f)
{
    if (!f) return;
    json_free(f->head);
    if (f->map) munmap(f->map, f->size);
    free(f);
}

int ckb_st_find(const CkbSafetensors *f, const char *name, CkbStTensor *out)
{
    const JsonValue *e = json_get(f->head, name), *shape = json_get(e, "shape"), *off = json_get(e, "data_offsets");
    if (!e || json_len(off) != 2 || json_len(shape) > 4) return 0;
    const double lo = json_num(json_at(off, 0), -1), hi = json_num(json_at(off, 1), -1);
    if (lo < 0 || hi < lo || hi > (double)(f->size - f->data0)) return 0;
    memset(out, 0, sizeof *out);
    out->dtype = json_str(json_get(e, "dtype"), "");
    out->ndim = json_len(shape);
    for (int i = 0; i < out->ndim; ++i) out->shape[i] = (long long)json_num(json_at(shape, i), -1);
    out->data = f->map + f->data0 + (size_t)lo;
    out->bytes = (size_t)(hi - lo);
    return 1;
}
