#include "cml_safetensors.h"

#include <fcntl.h>
#include <stdlib.h>
#include <string.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include "cml_internal.h"
#include "cml_json.h"

struct CMLSafetensors {
    uint8_t* map;
    size_t size, data_at;
    CMLJson* header;
};

CMLSafetensors* cml_safetensors_open(const char* path) {
    CMLSafetensors* st = NULL;
    struct stat sb;
    const int fd = open(path, O_RDONLY);
    if (fd < 0) { LOG_ERROR("cml_safetensors_open: cannot open '%s'", path); return NULL; }
    if (!fstat(fd, &sb) && sb.st_size > 8 && (st = (CMLSafetensors*)calloc(1, sizeof *st))) {
        st->size = (size_t)sb.st_size;
        void* m = mmap(NULL, st->size, PROT_READ, MAP_PRIVATE, fd, 0);
        if (m != MAP_FAILED) {
            st->map = (uint8_t*)m;
            uint64_t n = 0;
            for (int i = 0; i < 8; i++) n |= (uint64_t)st->map[i] << (8 * i);
            if (n <= st->size - 8) {
                st->header = cml_json_parse((const char*)st->map + 8, (size_t)n);
                st->data_at = 8 + (size_t)n;
            }
        }
    }
    close(fd);
    if (!st || !st->header || st->header->type != CML_JSON_OBJECT) {
        LOG_ERROR("cml_safetensors_open: '%s' is not a safetensors file", path);
        cml_safetensors_close(st);
        return NULL;
    }
    return st;
}

void cml_safetensors_close(CMLSafetensors* st) {
    if (!st) return;
    cml_json_free(st->header);
    if (st->map) munmap(st->map, st->size);
    free(st);
}

int cml_safetensors_find(const CMLSafetensors* st, const char* name, CMLSafetensor* out) {
    const CMLJson *e = st ? cml_json_get(st->header, name) : NULL, *shape = cml_json_get(e, "shape"), *off = cml_json_get(e, "data_offsets");
    const char* dt = cml_json_string(e, "dtype");
    if (!e) return -1;
    if (!dt || !shape || shape->type != CML_JSON_ARRAY || shape->count > 8 || !off || off->type != CML_JSON_ARRAY || off->count != 2) goto bad;
    memset(out, 0, sizeof *out);
    size_t esz;
    if (!strcmp(dt, "BF16")) { out->dtype = DTYPE_BFLOAT16; esz = 2; }
    else if (!strcmp(dt, "F16")) { out->dtype = DTYPE_FLOAT16; esz = 2; }
    else if (!strcmp(dt, "F32")) { out->dtype = DTYPE_FLOAT32; esz = 4; }
    else if (!strcmp(dt, "I32")) { out->dtype = DTYPE_INT32; esz = 4; }
    else goto bad;
    double numel = 1.0;
    for (const CMLJson* d = shape->child; d; d = d->next) {
        if (d->type != CML_JSON_NUMBER || d->number < 0 || d->number > 1e12) goto bad;
        out->shape[out->ndim++] = (int64_t)d->number;
        numel *= d->number;
    }
    const double a = off->child->number, b = off->child->next->number;
    if (a < 0 || b < a || b > (double)(st->size - st->data_at) || b - a != numel * (double)esz) goto bad;
    out->data = st->map + st->data_at + (size_t)a;
    out->bytes = (size_t)(b - a);
    return 0;
bad:
    LOG_ERROR("cml_safetensors_find: the entry of '%s' is malformed", name);
    return -1;
}
