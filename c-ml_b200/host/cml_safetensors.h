/* Reader of safetensors files: an 8-byte little-endian header length, that many bytes of JSON
 * (name -> dtype, shape, data_offsets into what follows), then the data. The file is mapped; a tensor's
 * bytes are checked to lie inside it and to match its shape. */
#ifndef CML_SAFETENSORS_H
#define CML_SAFETENSORS_H

#include <stddef.h>
#include <stdint.h>

#include "cml_quant_api.h"

typedef struct CMLSafetensors CMLSafetensors;
typedef struct CMLSafetensor {
    DType dtype;                 /* DTYPE_BFLOAT16, DTYPE_FLOAT16, DTYPE_FLOAT32 or DTYPE_INT32 */
    int ndim;
    int64_t shape[8];
    const void* data;            /* inside the mapping */
    size_t bytes;
} CMLSafetensor;

CMLSafetensors* cml_safetensors_open(const char* path);
void cml_safetensors_close(CMLSafetensors* st);
int cml_safetensors_find(const CMLSafetensors* st, const char* name, CMLSafetensor* out);      /* -1: absent or malformed */

#endif
