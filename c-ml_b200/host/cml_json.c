/* A recursive-descent JSON reader (RFC 8259) with a bound on the nesting depth. */
#include "cml_json.h"

#include <math.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>

#define MAX_DEPTH 64

typedef struct { const char *p, *end; } Cursor;

static void skip_blanks(Cursor* c) {
    while (c->p < c->end && (*c->p == ' ' || *c->p == '\t' || *c->p == '\n' || *c->p == '\r')) c->p++;
}

static int hex4(const char* s, unsigned* out) {
    unsigned v = 0;
    for (int i = 0; i < 4; i++) {
        const char ch = s[i];
        unsigned d;
        if (ch >= '0' && ch <= '9') d = (unsigned)(ch - '0');
        else if (ch >= 'a' && ch <= 'f') d = (unsigned)(ch - 'a' + 10);
        else if (ch >= 'A' && ch <= 'F') d = (unsigned)(ch - 'A' + 10);
        else return -1;
        v = v * 16 + d;
    }
    *out = v;
    return 0;
}

static char* put_utf8(char* o, unsigned u) {
    if (u < 0x80) *o++ = (char)u;
    else if (u < 0x800) { *o++ = (char)(0xC0 | (u >> 6)); *o++ = (char)(0x80 | (u & 63)); }
    else if (u < 0x10000) { *o++ = (char)(0xE0 | (u >> 12)); *o++ = (char)(0x80 | ((u >> 6) & 63)); *o++ = (char)(0x80 | (u & 63)); }
    else { *o++ = (char)(0xF0 | (u >> 18)); *o++ = (char)(0x80 | ((u >> 12) & 63)); *o++ = (char)(0x80 | ((u >> 6) & 63)); *o++ = (char)(0x80 | (u & 63)); }
    return o;
}

/* the cursor stands behind the opening quote */
static char* read_string(Cursor* c) {
    const char* q = c->p;
    while (q < c->end && *q != '"') q += (*q == '\\') ? 2 : 1;
    if (q >= c->end) return NULL;
    char* s = (char*)malloc((size_t)(q - c->p) + 1);     /* an escape never grows */
    if (!s) return NULL;
    char* o = s;
    const char* p = c->p;
    while (p < q) {
        if ((unsigned char)*p < 0x20) goto bad;
        if (*p != '\\') { *o++ = *p++; continue; }
        p++;
        switch (*p++) {
            case '"': *o++ = '"'; break;
            case '\\': *o++ = '\\'; break;
            case '/': *o++ = '/'; break;
            case 'b': *o++ = '\b'; break;
            case 'f': *o++ = '\f'; break;
            case 'n': *o++ = '\n'; break;
            case 'r': *o++ = '\r'; break;
            case 't': *o++ = '\t'; break;
            case 'u': {
                unsigned u, v;
                if (q - p < 4 || hex4(p, &u)) goto bad;
                p += 4;
                if (u >= 0xD800 && u < 0xDC00) {
                    if (q - p < 6 || p[0] != '\\' || p[1] != 'u' || hex4(p + 2, &v) || v < 0xDC00 || v > 0xDFFF) goto bad;
                    p += 6;
                    u = 0x10000 + ((u - 0xD800) << 10) + (v - 0xDC00);
                }
                o = put_utf8(o, u);
                break;
            }
            default: goto bad;
        }
    }
    *o = 0;
    c->p = q + 1;
    return s;
bad:
    free(s);
    return NULL;
}

static CMLJson* read_value(Cursor* c, int depth);

static CMLJson* read_members(Cursor* c, int depth, CMLJson* node, char close) {
    CMLJson** tail = &node->child;
    skip_blanks(c);
    if (c->p < c->end && *c->p == close) { c->p++; return node; }
    for (;;) {
        char* key = NULL;
        skip_blanks(c);
        if (node->type == CML_JSON_OBJECT) {
            if (c->p >= c->end || *c->p++ != '"' || !(key = read_string(c))) goto bad;
            skip_blanks(c);
            if (c->p >= c->end || *c->p++ != ':') { free(key); goto bad; }
        }
        CMLJson* v = read_value(c, depth + 1);
        if (!v) { free(key); goto bad; }
        v->key = key;
        *tail = v;
        tail = &v->next;
        node->count++;
        skip_blanks(c);
        if (c->p >= c->end) goto bad;
        const char ch = *c->p++;
        if (ch == close) return node;
        if (ch != ',') goto bad;
    }
bad:
    cml_json_free(node);
    return NULL;
}

static int word(Cursor* c, const char* w) {
    const size_t n = strlen(w);
    if ((size_t)(c->end - c->p) < n || memcmp(c->p, w, n)) return 0;
    c->p += n;
    return 1;
}

static CMLJson* read_value(Cursor* c, int depth) {
    skip_blanks(c);
    if (c->p >= c->end || depth > MAX_DEPTH) return NULL;
    CMLJson* n = (CMLJson*)calloc(1, sizeof *n);
    if (!n) return NULL;
    const char ch = *c->p;
    if (ch == '{' || ch == '[') {
        c->p++;
        n->type = ch == '{' ? CML_JSON_OBJECT : CML_JSON_ARRAY;
        return read_members(c, depth, n, ch == '{' ? '}' : ']');
    }
    if (ch == '"') {
        c->p++;
        n->type = CML_JSON_STRING;
        if ((n->string = read_string(c))) return n;
    } else if (word(c, "true")) { n->type = CML_JSON_BOOL; n->number = 1.0; return n; }
    else if (word(c, "false")) { n->type = CML_JSON_BOOL; return n; }
    else if (word(c, "null")) return n;
    else if (ch == '-' || (ch >= '0' && ch <= '9')) {
        char buf[64];
        size_t k = 0;
        while (c->p < c->end && k + 1 < sizeof buf && strchr("+-0123456789.eE", *c->p) && *c->p) buf[k++] = *c->p++;
        buf[k] = 0;
        char* stop;
        n->type = CML_JSON_NUMBER;
        n->number = strtod(buf, &stop);
        if (stop == buf + k && isfinite(n->number)) return n;
    }
    cml_json_free(n);
    return NULL;
}

CMLJson* cml_json_parse(const char* text, size_t len) {
    if (!text) return NULL;
    Cursor c = {text, text + len};
    CMLJson* n = read_value(&c, 0);
    skip_blanks(&c);
    if (n && c.p != c.end) { cml_json_free(n); return NULL; }
    return n;
}

CMLJson* cml_json_parse_file(const char* path) {
    FILE* f = fopen(path, "rb");
    if (!f) return NULL;
    CMLJson* j = NULL;
    char* text = NULL;
    if (!fseek(f, 0, SEEK_END)) {
        const long n = ftell(f);
        if (n > 0 && n < (1L << 28) && !fseek(f, 0, SEEK_SET) && (text = (char*)malloc((size_t)n)) && fread(text, 1, (size_t)n, f) == (size_t)n)
            j = cml_json_parse(text, (size_t)n);
    }
    free(text);
    fclose(f);
    return j;
}

void cml_json_free(CMLJson* j) {
    while (j) {
        CMLJson* next = j->next;
        cml_json_free(j->child);
        free(j->string);
        free(j->key);
        free(j);
        j = next;
    }
}

const CMLJson* cml_json_get(const CMLJson* object, const char* key) {
    if (!object || object->type != CML_JSON_OBJECT) return NULL;
    for (const CMLJson* c = object->child; c; c = c->next)
        if (!strcmp(c->key, key)) return c;
    return NULL;
}

int cml_json_double(const CMLJson* object, const char* key, double* out) {
    const CMLJson* v = cml_json_get(object, key);
    if (!v || v->type != CML_JSON_NUMBER) return -1;
    *out = v->number;
    return 0;
}

int cml_json_int(const CMLJson* object, const char* key, int* out) {
    double d;
    if (cml_json_double(object, key, &d) || d != floor(d) || fabs(d) > 2147483647.0) return -1;
    *out = (int)d;
    return 0;
}

const char* cml_json_string(const CMLJson* object, const char* key) {
    const CMLJson* v = cml_json_get(object, key);
    return v && v->type == CML_JSON_STRING ? v->string : NULL;
}
