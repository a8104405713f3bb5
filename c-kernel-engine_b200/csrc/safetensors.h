/* Read access to a safetensors file: 8-byte little-endian header length, a JSON header name -> {dtype, shape, data_offsets}, the data. */
#ifndef CKB200_SAFETENSORS_H
#define CKB200_SAFETENSORS_H

#include <stddef.h>
#include <stdint.h>

typedef struct CkbSafetensors CkbSafetensors;

typedef struct {
    const char *dtype;          /* "BF16", "I32", ... */
    int ndim;
    long long shape[4];
    const void *data;
    size_t bytes;
} CkbStTensor;

CkbSafetensors *ckb_st_open(const char *path);                              /* NULL on failure (error recorded) */
void ckb_st_close(CkbSafetensors *f);
int ckb_st_find(const CkbSafetensors *f, const char *name, CkbStTensor *out);   /* 1 when present */

#endif
