/* A small JSON reader: configuration files, safetensors headers and the step lines of a trace. The whole
 * text becomes a tree of nodes; every accessor takes NULL and the wrong kind of node. */
#ifndef CML_JSON_H
#define CML_JSON_H

#include <stddef.h>
#include <stdint.h>

typedef enum { CML_JSON_NULL, CML_JSON_BOOL, CML_JSON_NUMBER, CML_JSON_STRING, CML_JSON_ARRAY, CML_JSON_OBJECT } CMLJsonType;
typedef struct CMLJson {
    CMLJsonType type;
    double number;               /* numbers, and 0 / 1 of a bool */
    char* string;
    char* key;                   /* name within the parent object */
    int count;                   /* children of an array or object */
    struct CMLJson *child, *next;
} CMLJson;

CMLJson* cml_json_parse(const char* text, size_t len);       /* NULL on a syntax error; trailing blanks are allowed */
CMLJson* cml_json_parse_file(const char* path);
void cml_json_free(CMLJson* j);
const CMLJson* cml_json_get(const CMLJson* object, const char* key);      /* NULL: not an object, no such key */
/* 0 and the value; -1 (value untouched) when the key is absent, null or of another kind */
int cml_json_int(const CMLJson* object, const char* key, int* out);       /* whole numbers within int */
int cml_json_double(const CMLJson* object, const char* key, double* out);
const char* cml_json_string(const CMLJson* object, const char* key);

#endif
